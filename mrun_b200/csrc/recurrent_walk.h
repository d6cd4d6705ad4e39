// The register-tiled walk of bonus and state-space scans (recurrent_walk.cu), called by the entry points in
// recurrent.cu.
#pragma once

#include <cuda_runtime.h>

enum : int { WALK_BONUS = 0, WALK_SSM = 1 };

struct WalkArgs {
    int mode;
    const void *q, *k, *v;          // rows of one matrix, `ld` elements apart: q, k [H / group, D], v [H, V]
    long ld;
    const float* a;                 // bonus: float32 [tokens, H * D], the decays' arguments
    const void* dt;                 // state space: [tokens, H] in the activation type, rows `lddt` apart
    long lddt;
    const float *bias, *a_log, *bonus;      // bonus scan: bias and bonus [H * D]; state space: bias and a_log [H]
    float *state, *out;             // [slots, H, D, V]; [tokens, H * V]
    const int *seg_q_start, *seg_slot;
    int group, H, D, V;
    int max_q_len;                  // the longest segment
    int stage;                      // tokens a stage (set at the launch)
};

// Whether the walk takes this scan (sizes, alignments).
bool walk_takes(const WalkArgs& w, int act_dtype);
int launch_walk(const WalkArgs& w, int act_dtype, int segments, cudaStream_t stream);
