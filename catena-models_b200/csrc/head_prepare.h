// What the head preparation kernel takes (head_prepare.cu); the Python binding fills the same record
// (kernels._HeadPrepareArgs).
#pragma once
#include <cuda_runtime.h>

struct HeadPrepareArgs {
    void* qkv;                   // [rows][ld]: q | k | v of every row, overwritten in place
    long long ld;
    const float* bias;           // [(QH + 2 KVH) * HD] or null
    const float *wq, *wk;        // [HD] or null: the head norms' weights
    const float* rate;           // [pairs]: angle of pair i = position * rate[i]; further pairs stay
    const void* v_first;         // [rows][ld_first] or null: value rows to mix in, head j's channels at j * HD1 (DV1 of them)
    long long ld_first;
    const float* lam;            // the share of v_first (one float on the device)
    const int *tok_pos, *tok_seq, *seq_slot, *seq_end;
    void* pool;                  // [2][pages][KVH][PAGE_TOKENS][HD] or null: no cache write
    long long pages;
    const int* ptab;
    long long ptab_stride;
    long long rows;
    int QH, KVH, HD, norm_dim, pairs, interleaved, ring;
    int DV, DV1, HD1;            // value channels of a head without padding, here and in v_first
    int vec_first;               // set by the entry point: v_first is read eight channels at a time
    float eps, mag;
};
