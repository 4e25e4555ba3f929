// What the kernels of linear attention with a decay per head share: the activation code of q, k, v, and
// what is done to q and k in float32 on their way into the recurrence.
#pragma once

#include "common.cuh"

#define LIGHT_ACT_NONE 0
#define LIGHT_ACT_SILU 1

// Rotation of q and k (table null: none): value i turns with value i + dims/2 by the angle of the token's
// position; the table holds (cos, sin) per position and pair.  k is multiplied by k_scale afterwards.
struct LightRot {
    const float2* table;
    int dims, positions;
    const int* token_pos;
    float k_scale;
    int* status;
};

// A position outside the table is recorded, and the token is left unrotated.
__device__ __forceinline__ bool light_position_ok(const LightRot& rot, int pos) {
    if (pos >= 0 && pos < rot.positions) return true;
    if (threadIdx.x == 0 && rot.status != nullptr) atomicOr(rot.status, BFI_STATUS_BAD_POSITION);
    return false;
}
