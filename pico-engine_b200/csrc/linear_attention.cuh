// What the kernels of linear attention share: the description of a call, the activation of the projections, the cut of a step's
// packed tokens into chunks, and the tile kernels' launchers.
#pragma once
#include "common.cuh"

#define LA_CHUNK 64

struct LAArgs {
    const void* proj; int ld, q_off, k_off, v_off;
    const void* qk; int qk_ld;                 // the rows q and k are read from (proj itself, or float32 rows of their own)
    const void* z; int z_ld;
    const float* head_decay;
    float inv_tau, q_scale;
    int act_qk, act_v;
    float* state; long long state_stride;
    const int* row_first; const int* row_lens; const int* slots;
    float* out;
    int B, H, D, Dv;
    float* chunk_state;      // [chunks, H, D, Dv]
    float* chunk_decay;      // [chunks, H, D]
    int max_chunks;
};

// silu of a projection.  FAST (the bfloat16 engine, whose projections carry 8 bits): 2^x and the reciprocal from the
// special-function unit, relative error about 2^-22; else the exact routines.  A block applies it to every q and k entry of
// its head for each of its tokens, so its cost is paid once per 32 columns of the state.
template <bool FAST>
__device__ __forceinline__ float la_act(float v, int act) {
    if (act != 1) return v;
    if (FAST) {
        float e, r;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-1.4426950408889634f * v));
        asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
        return v * r;
    }
    return v / (1.0f + expf(-v));
}

// Which sequence chunk `c` of the step belongs to, its first packed token and its number of tokens (0: no such chunk).
__device__ __forceinline__ void la_find_chunk(const int* row_first, const int* row_lens, int B, int c, int& row, int& first, int& count) {
    int base = 0;
    row = -1; first = 0; count = 0;
    for (int b = 0; b < B; ++b) {
        const int n = row_lens[b], nc = (n + LA_CHUNK - 1) / LA_CHUNK;
        if (c < base + nc) {
            const int local = c - base;
            row = b; first = row_first[b] + local * LA_CHUNK;
            count = min(LA_CHUNK, n - local * LA_CHUNK);
            return;
        }
        base += nc;
    }
}

// Prompts with a decay per head, as products of tiles (linear_attention_tiles.cu): every chunk's contribution to the state, and, once
// each chunk's incoming state stands where its contribution was, every chunk's outputs.  `types`: 0 float32; 1 bfloat16 rows;
// 2 bfloat16 rows with float32 queries and keys of their own.
int la_tiles_contributions(const LAArgs& a, int types, cudaStream_t s);
int la_tiles_outputs(const LAArgs& a, int types, cudaStream_t s);
