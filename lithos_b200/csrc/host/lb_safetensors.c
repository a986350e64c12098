/* safetensors reader.  A file is a u64 LE header length, that many bytes of JSON ({"<name>": {"dtype": .., "shape": [..],
 * "data_offsets": [b, e]}, ..., "__metadata__": {..}}), then the data; offsets are relative to the end of the header. */
#define _GNU_SOURCE
#include "lb_internal.h"
#include "lb_json.h"
#include "lb_safetensors.h"
#include <dirent.h>
#include <errno.h>
#include <fcntl.h>
#include <stdarg.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

static int sfail(char* err, size_t errlen, int status, const char* fmt, ...) {
    if (err && errlen) {
        va_list ap;
        va_start(ap, fmt);
        vsnprintf(err, errlen, fmt, ap);
        va_end(ap);
    }
    return status;
}

/* map a whole file read-only (private); *bytes receives its size */
unsigned char* lb_map_file(const char* path, size_t* bytes) {
    int fd = open(path, O_RDONLY);
    if (fd < 0) return NULL;
    struct stat st;
    if (fstat(fd, &st) != 0 || st.st_size <= 0) { close(fd); return NULL; }
    void* p = mmap(NULL, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
    close(fd);
    if (p == MAP_FAILED) return NULL;
    *bytes = (size_t)st.st_size;
    return (unsigned char*)p;
}

static int cmp_tensor(const void* a, const void* b) { return strcmp(((const lb_st_tensor*)a)->name, ((const lb_st_tensor*)b)->name); }
static int cmp_str(const void* a, const void* b) { return strcmp(*(const char* const*)a, *(const char* const*)b); }

static int add_file(lb_st_set* s, int f, size_t* cap, char* err, size_t errlen) {
    const unsigned char* m = s->map[f];
    const size_t bytes = s->bytes[f];
    uint64_t hlen = 0;
    if (bytes >= 8) memcpy(&hlen, m, 8);
    if (bytes < 8 || hlen > bytes - 8)
        return sfail(err, errlen, LB_ERR_IO, "%s: header length %llu does not fit the file", s->file[f], (unsigned long long)hlen);
    char why[160];
    lb_json* j = lb_json_parse((const char*)m + 8, (size_t)hlen, why, sizeof why);
    if (!j || j->type != LB_JSON_OBJECT) {
        lb_json_free(j);
        return sfail(err, errlen, LB_ERR_IO, "%s: malformed header (%s)", s->file[f], j ? "not a JSON object" : why);
    }
    int st = LB_OK;
    for (int i = 0; i < j->n && st == LB_OK; i++) {
        if (!strcmp(j->key[i], "__metadata__")) continue;
        const lb_json *v = &j->item[i], *o = lb_json_get(v, "data_offsets"), *sh = lb_json_get(v, "shape");
        const char* dt = lb_json_str(v, "dtype");
        const double lim = (double)(bytes - 8 - hlen);
        if (!o || o->type != LB_JSON_ARRAY || o->n != 2 || !(o->item[0].num >= 0) || !(o->item[1].num >= o->item[0].num) || !(o->item[1].num <= lim)) {
            st = sfail(err, errlen, LB_ERR_IO, "%s: tensor %s has no valid data_offsets", s->file[f], j->key[i]);
            break;
        }
        if (s->n == *cap) {
            const size_t c2 = *cap ? *cap * 2 : 1024;
            lb_st_tensor* t = (lb_st_tensor*)realloc(s->t, c2 * sizeof *t);
            if (!t) { st = sfail(err, errlen, LB_ERR_NOMEM, "safetensors: out of memory"); break; }
            s->t = t;
            *cap = c2;
        }
        lb_st_tensor* t = &s->t[s->n];
        memset(t, 0, sizeof *t);
        t->name = strdup(j->key[i]);
        if (!t->name) { st = sfail(err, errlen, LB_ERR_NOMEM, "safetensors: out of memory"); break; }
        if (dt) snprintf(t->dtype, sizeof t->dtype, "%s", dt);
        t->ndim = -1; /* unknown, or more dimensions than this reader describes */
        if (sh && sh->type == LB_JSON_ARRAY && sh->n <= LB_ST_MAX_DIMS) {
            t->ndim = sh->n;
            for (int d = 0; d < sh->n; d++) t->dim[d] = (int64_t)sh->item[d].num;
        }
        t->file = (uint32_t)f;
        t->off = 8 + hlen + (uint64_t)o->item[0].num;
        t->size = (uint64_t)o->item[1].num - (uint64_t)o->item[0].num;
        t->data = m + t->off;
        s->n++;
    }
    lb_json_free(j);
    return st;
}

int lb_st_open(const char* dir, lb_st_set* s, char* err, size_t errlen) {
    memset(s, 0, sizeof *s);
    DIR* d = opendir(dir);
    if (!d) return sfail(err, errlen, LB_ERR_IO, "cannot open %s (%s)", dir, strerror(errno));
    int st = LB_OK;
    for (struct dirent* e; (e = readdir(d)) != NULL;) {
        const size_t n = strlen(e->d_name);
        if (n < 13 || n > 255 || strcmp(e->d_name + n - 12, ".safetensors")) continue;
        if (s->n_files == LB_ST_MAX_FILES) { st = sfail(err, errlen, LB_ERR_IO, "%s holds more than %d safetensors files", dir, LB_ST_MAX_FILES); break; }
        s->file[s->n_files++] = strdup(e->d_name);
    }
    closedir(d);
    if (st == LB_OK && !s->n_files) st = sfail(err, errlen, LB_ERR_IO, "%s holds no *.safetensors file", dir);
    qsort(s->file, (size_t)s->n_files, sizeof s->file[0], cmp_str);
    size_t cap = 0;
    for (int i = 0; i < s->n_files && st == LB_OK; i++) {
        char path[1536];
        snprintf(path, sizeof path, "%s/%s", dir, s->file[i]);
        s->map[i] = lb_map_file(path, &s->bytes[i]);
        st = s->map[i] ? add_file(s, i, &cap, err, errlen) : sfail(err, errlen, LB_ERR_IO, "cannot map %s (%s)", path, strerror(errno));
    }
    if (st == LB_OK) qsort(s->t, s->n, sizeof *s->t, cmp_tensor);
    else lb_st_close(s);
    return st;
}

void lb_st_close(lb_st_set* s) {
    for (int i = 0; i < s->n_files; i++) {
        if (s->map[i]) munmap(s->map[i], s->bytes[i]);
        free(s->file[i]);
    }
    for (size_t i = 0; i < s->n; i++) free(s->t[i].name);
    free(s->t);
    memset(s, 0, sizeof *s);
}

const lb_st_tensor* lb_st_find(const lb_st_set* s, const char* name) {
    lb_st_tensor key;
    key.name = (char*)name;
    return s->n ? (const lb_st_tensor*)bsearch(&key, s->t, s->n, sizeof *s->t, cmp_tensor) : NULL;
}
