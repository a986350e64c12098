/* A small JSON reader (config.json, safetensors headers): parsed into a tree that one call frees. */
#ifndef LB_JSON_H
#define LB_JSON_H
#include <stddef.h>

enum { LB_JSON_NULL, LB_JSON_BOOL, LB_JSON_NUMBER, LB_JSON_STRING, LB_JSON_ARRAY, LB_JSON_OBJECT };
typedef struct lb_json {
    int type;
    double num;           /* number, or 0 / 1 of a boolean */
    char* str;            /* string (UTF-8, escapes decoded) */
    int n;                /* elements / members */
    struct lb_json* item; /* [n] */
    char** key;           /* [n] of an object */
} lb_json;

/* NULL on malformed text (err says where) or when memory runs out */
lb_json* lb_json_parse(const char* text, size_t len, char* err, size_t errlen);
void lb_json_free(lb_json* j);
const lb_json* lb_json_get(const lb_json* j, const char* key);              /* member of an object, or NULL */
int lb_json_has(const lb_json* j, const char* key);                          /* the member exists and is not null */
double lb_json_num(const lb_json* j, const char* key, double missing);       /* number member, else `missing` */
const char* lb_json_str(const lb_json* j, const char* key);                  /* string member, else NULL */
#endif
