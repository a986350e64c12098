/* JSON reader: recursive descent over the text, no dependencies. */
#include "lb_json.h"
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#define JSON_MAX_DEPTH 64

typedef struct { const char *p, *end, *begin; const char* what; } jp;

static void ws(jp* s) { while (s->p < s->end && (*s->p == ' ' || *s->p == '\n' || *s->p == '\t' || *s->p == '\r')) s->p++; }
static int bad(jp* s, const char* what) { if (!s->what) s->what = what; return 0; }

static void put_utf8(char** o, unsigned c) {
    unsigned char* q = (unsigned char*)*o;
    if (c < 0x80) *q++ = (unsigned char)c;
    else if (c < 0x800) { *q++ = (unsigned char)(0xC0 | c >> 6); *q++ = (unsigned char)(0x80 | (c & 63)); }
    else if (c < 0x10000) { *q++ = (unsigned char)(0xE0 | c >> 12); *q++ = (unsigned char)(0x80 | (c >> 6 & 63)); *q++ = (unsigned char)(0x80 | (c & 63)); }
    else { *q++ = (unsigned char)(0xF0 | c >> 18); *q++ = (unsigned char)(0x80 | (c >> 12 & 63)); *q++ = (unsigned char)(0x80 | (c >> 6 & 63)); *q++ = (unsigned char)(0x80 | (c & 63)); }
    *o = (char*)q;
}
static int hex4(jp* s, unsigned* v) {
    if (s->end - s->p < 4) return 0;
    *v = 0;
    for (int i = 0; i < 4; i++) {
        const char c = *s->p++;
        const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
        if (d < 0) return 0;
        *v = *v << 4 | (unsigned)d;
    }
    return 1;
}
static char* string(jp* s) {
    if (s->p >= s->end || *s->p != '"') { bad(s, "a string was expected"); return NULL; }
    const char* q = ++s->p;
    while (q < s->end && *q != '"') q += *q == '\\' ? 2 : 1;
    if (q >= s->end) { bad(s, "unterminated string"); return NULL; }
    char *out = (char*)malloc((size_t)(q - s->p) + 1), *o = out; /* decoded text is never longer */
    if (!out) { bad(s, "out of memory"); return NULL; }
    while (s->p < q) {
        if (*s->p != '\\') { *o++ = *s->p++; continue; }
        const char c = s->p[1];
        s->p += 2;
        const char* from = "\"\\/bfnrt"; const char* to = "\"\\/\b\f\n\r\t";
        const char* f = c ? strchr(from, c) : NULL;
        if (f) { *o++ = to[f - from]; continue; }
        unsigned u, lo;
        if (c != 'u' || !hex4(s, &u)) { free(out); bad(s, "bad escape"); return NULL; }
        if (u >= 0xD800 && u < 0xDC00 && s->end - s->p >= 6 && s->p[0] == '\\' && s->p[1] == 'u') {
            s->p += 2;
            if (!hex4(s, &lo)) { free(out); bad(s, "bad escape"); return NULL; }
            u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
        }
        put_utf8(&o, u);
    }
    *o = 0;
    s->p = q + 1;
    return out;
}

static void release(lb_json* j) {
    for (int i = 0; i < j->n; i++) {
        if (j->item) release(&j->item[i]);
        if (j->key) free(j->key[i]);
    }
    free(j->item); free(j->key); free(j->str);
    memset(j, 0, sizeof *j);
}

static int value(jp* s, lb_json* j, int depth);

static int container(jp* s, lb_json* j, int depth, char close) {
    int cap = 0;
    s->p++;
    ws(s);
    if (s->p < s->end && *s->p == close) { s->p++; return 1; }
    for (;;) {
        if (j->n == cap) {
            const int c2 = cap ? cap * 2 : 8;
            lb_json* it = (lb_json*)realloc(j->item, (size_t)c2 * sizeof *it);
            if (!it) return bad(s, "out of memory");
            j->item = it;
            if (close == '}') {
                char** k = (char**)realloc(j->key, (size_t)c2 * sizeof *k);
                if (!k) return bad(s, "out of memory");
                j->key = k;
            }
            cap = c2;
        }
        memset(&j->item[j->n], 0, sizeof *j->item);
        if (close == '}') {
            ws(s);
            char* k = string(s);
            if (!k) return 0;
            j->key[j->n] = k;
            j->n++;
            ws(s);
            if (s->p >= s->end || *s->p != ':') return bad(s, "':' was expected");
            s->p++;
        } else j->n++;
        if (!value(s, &j->item[j->n - 1], depth + 1)) return 0;
        ws(s);
        if (s->p < s->end && *s->p == ',') { s->p++; continue; }
        if (s->p < s->end && *s->p == close) { s->p++; return 1; }
        return bad(s, "',' or the end of a list was expected");
    }
}

static int value(jp* s, lb_json* j, int depth) {
    ws(s);
    if (s->p >= s->end) return bad(s, "unexpected end");
    if (depth > JSON_MAX_DEPTH) return bad(s, "nested too deeply");
    const size_t left = (size_t)(s->end - s->p);
    if (*s->p == '{') { j->type = LB_JSON_OBJECT; return container(s, j, depth, '}'); }
    if (*s->p == '[') { j->type = LB_JSON_ARRAY; return container(s, j, depth, ']'); }
    if (*s->p == '"') { j->type = LB_JSON_STRING; return (j->str = string(s)) != NULL; }
    if (left >= 4 && !memcmp(s->p, "null", 4)) { s->p += 4; return 1; }
    if (left >= 4 && !memcmp(s->p, "true", 4)) { s->p += 4; j->type = LB_JSON_BOOL; j->num = 1; return 1; }
    if (left >= 5 && !memcmp(s->p, "false", 5)) { s->p += 5; j->type = LB_JSON_BOOL; return 1; }
    char num[64]; /* a terminated copy: the text may be a slice of a mapped file */
    size_t n = 0;
    while (n < left && n < sizeof num - 1 && strchr("+-0123456789.eE", s->p[n]) && s->p[n]) { num[n] = s->p[n]; n++; }
    num[n] = 0;
    char* e = NULL;
    j->num = n ? strtod(num, &e) : 0;
    if (!n || e != num + n) return bad(s, "a value was expected");
    j->type = LB_JSON_NUMBER;
    s->p += n;
    return 1;
}

lb_json* lb_json_parse(const char* text, size_t len, char* err, size_t errlen) {
    jp s = {text, text + len, text, NULL};
    lb_json* j = (lb_json*)calloc(1, sizeof *j);
    if (!j) return NULL;
    int ok = value(&s, j, 0);
    if (ok) {
        while (s.p < s.end && (*s.p == ' ' || *s.p == '\n' || *s.p == '\t' || *s.p == '\r' || *s.p == 0)) s.p++;
        if (s.p < s.end) ok = bad(&s, "text after the value");
    }
    if (ok) return j;
    if (err) snprintf(err, errlen, "malformed JSON at byte %zu: %s", (size_t)(s.p - s.begin), s.what ? s.what : "?");
    lb_json_free(j);
    return NULL;
}
void lb_json_free(lb_json* j) {
    if (!j) return;
    release(j);
    free(j);
}
const lb_json* lb_json_get(const lb_json* j, const char* key) {
    if (j && j->type == LB_JSON_OBJECT)
        for (int i = 0; i < j->n; i++)
            if (!strcmp(j->key[i], key)) return &j->item[i];
    return NULL;
}
int lb_json_has(const lb_json* j, const char* key) {
    const lb_json* v = lb_json_get(j, key);
    return v && v->type != LB_JSON_NULL;
}
double lb_json_num(const lb_json* j, const char* key, double missing) {
    const lb_json* v = lb_json_get(j, key);
    return v && v->type == LB_JSON_NUMBER ? v->num : missing;
}
const char* lb_json_str(const lb_json* j, const char* key) {
    const lb_json* v = lb_json_get(j, key);
    return v && v->type == LB_JSON_STRING ? v->str : NULL;
}
