/* safetensors files of a directory, mapped read-only, their tensors by name. */
#ifndef LB_SAFETENSORS_H
#define LB_SAFETENSORS_H
#include <stddef.h>
#include <stdint.h>

#define LB_ST_MAX_FILES 64
#define LB_ST_MAX_DIMS 4
typedef struct {
    char* name;
    char dtype[8]; /* as in the header: BF16, F16, F32, I32, ... */
    int ndim;
    int64_t dim[LB_ST_MAX_DIMS];
    uint32_t file;
    uint64_t off, size; /* inside the file */
    const void* data;
} lb_st_tensor;
typedef struct {
    int n_files;
    char* file[LB_ST_MAX_FILES];
    unsigned char* map[LB_ST_MAX_FILES];
    size_t bytes[LB_ST_MAX_FILES];
    lb_st_tensor* t; /* in name order */
    size_t n;
} lb_st_set;

int lb_st_open(const char* dir, lb_st_set* out, char* err, size_t errlen); /* every *.safetensors file of dir, in name order */
void lb_st_close(lb_st_set* s);
const lb_st_tensor* lb_st_find(const lb_st_set* s, const char* name);
#endif
