// Argument block shared by every matrix-product kernel of the engine.
//
//   C[c_row(i), n] (=|+=) epilogue( sum_k A[a_row(i), k] * W[g(i)][n, k] )      i in [0, M)
//
// A is [rows, K] with leading dimension lda; W is [groups][N (or 2N), K], row-major
// ("out, in"), groups `w_group_stride` elements apart.  Logical rows are split
// among the groups by `group_offsets[0..n_groups]` (ascending; rows of group g are
// [off[g], off[g+1])); with no offsets there is one group.  `a_rows` gathers the
// rows of A, `c_rows` scatters the rows of C; either may be null (identity).
// `row_scale`, if given, is indexed by a_row(i) when `scale_by_a_row` else by i.
#pragma once
#include "common.cuh"

enum GemmEpilogue {
    EPI_STORE = 0,        // C (activation type) = act(acc * scale), act by `activation`
    EPI_STORE_F32 = 1,    // C (float32) = acc * scale
    EPI_ADD_F32 = 2,      // C (float32) += acc * scale          (residual stream)
    EPI_SWIGLU = 3        // C (activation type) = act(s*gate) * (s*up), act by `activation`: silu, or gelu if it says so;
                          // W rows [0,N) gate, [N,2N) up
};

struct GemmParams {
    const void* A;
    const void* W;
    void* C;
    const int* a_rows;
    const int* c_rows;
    const int* group_offsets;
    const float* row_scale;
    long long lda, ldc, w_group_stride;
    int n_groups, M, N, K;
    int epilogue;
    int scale_by_a_row;
    int activation;       // SPITE_ACT_*: applied by EPI_STORE to the scaled sum (plus bias) before it is rounded; with EPI_SWIGLU
                          // the gate's: SPITE_ACT_NONE (silu) or SPITE_ACT_GELU_TANH
    const float* bias;    // [N] or null: added by EPI_STORE to the scaled sum before the activation (one group)
    float act_pos, act_neg;   // SPITE_ACT_XIELU: the coefficients of its two branches
};

#define SPITE_ACT_NONE 0
#define SPITE_ACT_RELU2 1        // relu(y)^2
#define SPITE_ACT_GELU_TANH 2    // 0.5 y (1 + tanh(sqrt(2/pi) (y + 0.044715 y^3)))
#define SPITE_ACT_XIELU 3        // y > 0: act_pos y^2 + y / 2; else act_neg (e^y - 1 - y) + y / 2
#define SPITE_ACT_TANH 4

__device__ __forceinline__ float gelu_tanh_f32(float y) {
    return 0.5f * y * (1.0f + tanhf(0.7978845608028654f * (y + 0.044715f * y * y * y)));
}
__device__ __forceinline__ float apply_activation(const GemmParams& p, float y) {
    const int act = p.activation;
    if (act == SPITE_ACT_RELU2) { y = fmaxf(y, 0.f); y *= y; }
    else if (act == SPITE_ACT_GELU_TANH) y = gelu_tanh_f32(y);
    else if (act == SPITE_ACT_XIELU) {
        const float n = fminf(y, 0.f);                       // (no branch per element)
        const float pos = fmaxf(y, 0.f);
        y = fmaf(p.act_pos * pos, pos, fmaf(p.act_neg, expm1f(n) - n, 0.5f * y));
    } else if (act == SPITE_ACT_TANH) y = tanhf(y);
    return y;
}
// The same for output column n: the bias first.
__device__ __forceinline__ float finish_store(const GemmParams& p, float y, int n) {
    return apply_activation(p, p.bias ? y + p.bias[n] : y);
}

// An activation goes with the plain store (the gated form takes gelu for its gate), a bias with the plain store of a product
// of one group.
static inline bool activation_ok(const GemmParams* p) {
    if (p->activation < SPITE_ACT_NONE || p->activation > SPITE_ACT_TANH) return false;
    if (p->bias && (p->epilogue != EPI_STORE || p->group_offsets)) return false;
    if (p->epilogue == EPI_SWIGLU && p->activation == SPITE_ACT_GELU_TANH) return true;
    return p->activation == SPITE_ACT_NONE || p->epilogue == EPI_STORE;
}

__device__ __forceinline__ float silu_f32(float g) { return g / (1.0f + expf(-g)); }
// The gated epilogue's factor: silu or gelu of the gate's sum.
__device__ __forceinline__ float gate_factor(const GemmParams& p, float g) {
    return p.activation == SPITE_ACT_GELU_TANH ? gelu_tanh_f32(g) : silu_f32(g);
}

// Finds the (group, first row, row count) of the `tile`-th row tile when every
// group is cut into tiles of `bm` rows of its own.  Returns false past the end.
__device__ __forceinline__ bool locate_row_tile(const GemmParams& p, int tile, int bm,
                                                int& group, int& row0, int& rows) {
    if (!p.group_offsets) {
        group = 0; row0 = tile * bm; rows = min(bm, p.M - row0);
        return row0 < p.M;
    }
    for (int g = 0; g < p.n_groups; ++g) {
        const int lo = p.group_offsets[g], hi = p.group_offsets[g + 1];
        const int tiles = (hi - lo + bm - 1) / bm;
        if (tile < tiles) { group = g; row0 = lo + tile * bm; rows = min(bm, hi - row0); return true; }
        tile -= tiles;
    }
    return false;
}
