// Recurrent mixers whose state is a matrix per head that decays and takes one outer product a token, carried from token to
// token in float32 in the request's state slot.  One walk serves three designs:
//
//   state space (Mamba-2):   dt = softplus(a + dt_bias),  S <- exp(-exp(A_log) dt) S + dt k v^T,   o = S^T q + D v
//                            (one decay a head and token; q and k shared by a group of heads; read after the write)
//   decaying memory (RWKV):  o = S^T q + (sum_i q_i u_i k_i) v,   S <- diag(w) S + k v^T,   w = exp(-exp(z + w0))
//                            (a decay per key channel; the token itself enters the read-out through the bonus u)
//   gated linear attention:  S <- diag(w) S + k v^T,   o = c S^T q,   w = sigmoid(z)^(1/tau),   z = A_2 a + b
//                            (a decay per key channel from a short vector a; read after the write)
//
// S is [dim keys, vdim values], zeros at the start of a sequence.  Everything is float32.
//
// Unlike a delta rule, what a token writes does not depend on the state, so the walk is bound by what its warps can issue,
// not by one token's chain.  A warp is LR lanes along the keys times 32 / LR lanes along the values; a lane holds 4 RPV
// key rows (as packed pairs, for the two-at-a-time multiply-adds of sm_100) of CC value columns.  TB tokens form a batch:
// one more warp of the block brings their inputs into one stage of a shared-memory ring by asynchronous copies three batches
// ahead (so that the walking warps spend nothing on it; its lanes keep the addresses of what they copy in registers), one barrier stands between two batches, and the batch's TB * CC
// partial read-outs a lane are summed over the LR lanes by a halving exchange that leaves every lane TB * CC / LR finished
// numbers.  The order of the sums depends on the head's sizes alone, so the result does not depend on how a sequence was
// cut into steps.
//
// The slot holds S transposed: value column j's keys are contiguous, [vdim, dim4] with dim4 = dim rounded up to a multiple
// of four (the padding stays zero), so that a lane's rows are whole 16-byte groups and a warp's loads whole lines.
#include "common.cuh"

struct ScanParams {
    const float* q; const float* k; const float* v;       // first element of token 0's q, k [kv_heads * dim], v [heads * vdim]
    long long q_stride, k_stride, v_stride;               // floats between two tokens' rows
    const float* w; long long w_stride;                   // decay per key channel [tokens, heads * dim], or null: per head
    const float* scalars;                                 // [tokens, heads, 4]: (decay, dt, -, -) without w; (bonus, -, -, -) with w;
                                                          // not read (null) by gated linear attention
    const float* skip;                                    // [heads] the factor D on v in the read-out, or null
    float* out; long long out_stride;                     // [tokens, heads * vdim]
    float* state; long long slot_stride;                  // state + slot * slot_stride + head * vdim * dim4
    const int* cu_seqlens; const int* slots;
    int n_segments, n_tokens, heads, kv_heads, dim, vdim;
    float out_scale;                                      // gated linear attention: the factor c on the read-out
};

namespace {

typedef unsigned long long f2;                            // two packed floats

__device__ __forceinline__ f2 pack2(float lo, float hi) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

constexpr int RING = 4;

constexpr int MAX_WARPS = 4;                              // walking warps a block

// the three designs
enum Walk { PER_HEAD = 0, PER_CHANNEL_BONUS = 1, PER_CHANNEL = 2 };

template <int LR, int RPV, int CC, int TB, int WALK>
struct Shape {
    static constexpr bool CH = WALK != PER_HEAD;          // a decay per key channel
    static constexpr bool SCALARS = WALK != PER_CHANNEL;  // a token brings scalars
    static constexpr int DP = LR * RPV * 4;               // key rows a warp covers
    static constexpr int WC = 32 / LR * CC;               // value columns a warp covers
    static constexpr int ROWS = CH ? 3 : 2;               // q, k (and w) of a token
    static constexpr int TOKEN = ROWS * DP + WC * MAX_WARPS + 4;      // floats of a token's stage
    static constexpr int KEEP = TB * CC / LR;             // finished numbers a lane
    static_assert(KEEP >= 1 && KEEP * LR == TB * CC && TOKEN % 4 == 0, "a batch's read-outs must fill the lanes");
};

// All threads of the block (the number is a multiple of 32).
__device__ __forceinline__ void block_barrier(int threads) { asm volatile("bar.sync 1, %0;" ::"r"(threads) : "memory"); }

// What one lane of the bringing warp copies of every token, in 16-byte groups (rows that are whole groups).
template <typename SH, int TB>
struct Bringer {
    static constexpr bool CH = SH::ROWS == 3;
    static constexpr int V = SH::ROWS * SH::DP;
    static constexpr int SLOTS = (SH::ROWS * (SH::DP / 4) + SH::WC * MAX_WARPS / 4 + 1 + 31) / 32;
    const float* src[SLOTS];
    long long stride[SLOTS];
    int dst[SLOTS];                                       // floats into a token's stage; < 0: nothing

    __device__ __forceinline__ Bringer(const ScanParams& p, const float* qp, const float* kp, const float* wp, const float* vp,
                                       const float* sp, int n_cols, long long t0, int lane) {
        const int du = p.dim >> 2, vu = n_cols >> 2, rows = SH::ROWS * du;
#pragma unroll
        for (int s = 0; s < SLOTS; ++s) {
            const int e = lane + 32 * s;
            src[s] = nullptr; stride[s] = 0; dst[s] = -1;
            if (e < du) { src[s] = qp + 4 * e; stride[s] = p.q_stride; dst[s] = 4 * e; }
            else if (e < 2 * du) { src[s] = kp + 4 * (e - du); stride[s] = p.k_stride; dst[s] = SH::DP + 4 * (e - du); }
            else if (CH && e < 3 * du) { src[s] = wp + 4 * (e - 2 * du); stride[s] = p.w_stride; dst[s] = 2 * SH::DP + 4 * (e - 2 * du); }
            else if (e < rows + vu) { src[s] = vp + 4 * (e - rows); stride[s] = p.v_stride; dst[s] = V + 4 * (e - rows); }
            else if (SH::SCALARS && e == rows + vu) { src[s] = sp; stride[s] = 4 * p.heads; dst[s] = SH::TOKEN - 4; }
            if (dst[s] >= 0) src[s] += t0 * stride[s];
        }
    }
    // the next n tokens into `stage`
    __device__ __forceinline__ void bring(float* stage, int n) {
#pragma unroll
        for (int s = 0; s < SLOTS; ++s) {
            if (dst[s] < 0) continue;
            float* d = stage + dst[s];
            if (n == TB) {
#pragma unroll
                for (int tt = 0; tt < TB; ++tt) { cp_async16(d + tt * SH::TOKEN, src[s]); src[s] += stride[s]; }
            } else {
                for (int tt = 0; tt < n; ++tt) { cp_async16(d + tt * SH::TOKEN, src[s]); src[s] += stride[s]; }
            }
        }
    }
};
// The same element by element, for rows of other lengths.
template <typename SH>
__device__ __forceinline__ void bring_elements(const ScanParams& p, const float* qp, const float* kp, const float* wp, const float* vp,
                                               const float* sp, int n_cols, long long tb, int n, float* stage, int lane) {
    constexpr bool CH = SH::ROWS == 3;
    constexpr int V = SH::ROWS * SH::DP;
    const int dim = p.dim;
#pragma unroll 1
    for (int tt = 0; tt < n; ++tt) {
        float* d = stage + tt * SH::TOKEN;
        const long long t = tb + tt;
        for (int e = lane; e < dim; e += 32) {
            cp_async4(d + e, qp + t * p.q_stride + e);
            cp_async4(d + SH::DP + e, kp + t * p.k_stride + e);
            if constexpr (CH) cp_async4(d + 2 * SH::DP + e, wp + t * p.w_stride + e);
        }
        for (int e = lane; e < n_cols; e += 32) cp_async4(d + V + e, vp + t * p.v_stride + e);
        if (SH::SCALARS && lane < 2) cp_async4(d + SH::TOKEN - 4 + lane, sp + t * (4 * p.heads) + lane);
    }
}

// grid (ceil(vdim / (WC * warps)), heads, segments), block 32 * (warps + 1)
template <int LR, int RPV, int CC, int TB, int WALK>
__global__ void __launch_bounds__(32 * (MAX_WARPS + 1)) scan_kernel(const ScanParams p, const int wide) {
    using SH = Shape<LR, RPV, CC, TB, WALK>;
    constexpr bool CH = SH::CH;
    constexpr int DP = SH::DP, WC = SH::WC, NP = RPV * 2, TOKEN = SH::TOKEN, V = SH::ROWS * DP;
    extern __shared__ __align__(16) float ring[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x >> 5) - 1;
    const int seg = blockIdx.z, head = blockIdx.y;
    const int dim = p.dim, vdim = p.vdim, dim4 = (dim + 3) & ~3;
    const int BC = WC * warps, c0 = blockIdx.x * BC;
    // rows beyond dim stay zero in every stage (a decay there multiplies zeros)
    if (DP > dim) {
        const int gap = DP - dim;
        for (int e = threadIdx.x; e < RING * TB * SH::ROWS * gap; e += blockDim.x) {
            const int t = e / (SH::ROWS * gap), i = e % (SH::ROWS * gap);
            ring[t * TOKEN + (i / gap) * DP + dim + i % gap] = 0.f;
        }
    }
    pdl_wait();
    const int t0 = p.cu_seqlens[seg], t1 = p.cu_seqlens[seg + 1];
    if (t0 >= t1) return;
    const int slot = p.slots[seg];
    if (seg > 0 && slot == p.slots[0]) {                  // a captured step's padding row (a copy of the first row): the state
        for (int e = threadIdx.x; e < (t1 - t0) * BC; e += blockDim.x)      // moves on once; the copy's results are never read
            if (c0 + e % BC < vdim) p.out[(size_t)(t0 + e / BC) * p.out_stride + (size_t)head * vdim + c0 + e % BC] = 0.f;
        return;
    }
    const int n_cols = min(BC, vdim - c0);
    const int n_batches = (t1 - t0 + TB - 1) / TB;

    if (warp == warps) {                                  // the warp that brings the inputs
        const int kvh = head / (p.heads / p.kv_heads);
        const float* qp = p.q + (size_t)kvh * dim;
        const float* kp = p.k + (size_t)kvh * dim;
        const float* vp = p.v + (size_t)head * vdim + c0;
        const float* wp = CH ? p.w + (size_t)head * dim : nullptr;
        const float* sp = SH::SCALARS ? p.scalars + 4 * head : nullptr;
        const auto pump = [&](auto&& bring) {             // bring(batch): starts its copies
#pragma unroll 1
            for (int b = 0; b < RING - 1; ++b) { bring(b); cp_commit(); }
#pragma unroll 1
            for (int b = 0; b < n_batches; ++b) {
                cp_wait<RING - 2>();
                block_barrier(blockDim.x);                // batch b has landed, and every warp is done with batch b - 1
                bring(b + RING - 1);                      // (into the stage that batch b - 1 had)
                cp_commit();
            }
            cp_wait<0>();
        };
        if (wide) {
            Bringer<SH, TB> br(p, qp, kp, wp, vp, sp, n_cols, t0, lane);
            pump([&](int b) { if (b < n_batches) br.bring(ring + (b % RING) * TB * TOKEN, min(TB, t1 - t0 - b * TB)); });
        } else {
            pump([&](int b) {
                if (b < n_batches)
                    bring_elements<SH>(p, qp, kp, wp, vp, sp, n_cols, t0 + (long long)b * TB, min(TB, t1 - t0 - b * TB),
                                       ring + (b % RING) * TB * TOKEN, lane);
            });
        }
        return;
    }

    // the state: value column j = c0 + warp * WC + cl * CC + c, key rows 4 (r + LR i) .. + 3
    const int r = lane % LR, cl = lane / LR;
    float* st = p.state + (size_t)slot * p.slot_stride + (size_t)head * vdim * dim4;
    const int j0 = warp * WC + cl * CC;                   // within the block's columns
    f2 S[NP][CC];
#pragma unroll
    for (int c = 0; c < CC; ++c)
#pragma unroll
        for (int i = 0; i < RPV; ++i) {
            const int row = 4 * (r + LR * i);
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            if (row < dim4 && j0 + c < n_cols) f = *(const float4*)(st + (size_t)(c0 + j0 + c) * dim4 + row);
            S[2 * i][c] = pack2(f.x, f.y); S[2 * i + 1][c] = pack2(f.z, f.w);
        }

    const float skip = p.skip ? p.skip[head] : 0.f;
    auto token = [&](const float* in, float* o) {         // in: the token's stage
        f2 q[NP], k[NP], w[CH ? NP : 1];
#pragma unroll
        for (int i = 0; i < RPV; ++i) {
            const int row = 4 * (r + LR * i);
            const ulonglong2 a = *(const ulonglong2*)(in + row), b = *(const ulonglong2*)(in + DP + row);
            q[2 * i] = a.x; q[2 * i + 1] = a.y; k[2 * i] = b.x; k[2 * i + 1] = b.y;
            if constexpr (CH) {
                const ulonglong2 d = *(const ulonglong2*)(in + 2 * DP + row);
                w[2 * i] = d.x; w[2 * i + 1] = d.y;
            }
        }
        f2 decay = 0;
        float v[CC];
        if constexpr (CC == 4) { const float4 f = *(const float4*)(in + V + j0); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
        else { const float2 f = *(const float2*)(in + V + j0); v[0] = f.x; v[1] = f.y; }
        if constexpr (!CH) {
            const float2 s = *(const float2*)(in + TOKEN - 4);
            decay = pack2(s.x, s.x);
#pragma unroll
            for (int c = 0; c < CC; ++c) v[c] *= s.y;
        }
#pragma unroll
        for (int c = 0; c < CC; ++c) {
            const f2 v2 = pack2(v[c], v[c]);
            f2 acc = 0;
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                if constexpr (WALK == PER_CHANNEL_BONUS) {
                    acc = fma2(q[i], S[i][c], acc);
                    S[i][c] = fma2(w[i], S[i][c], mul2(k[i], v2));
                } else if constexpr (WALK == PER_CHANNEL) {
                    S[i][c] = fma2(w[i], S[i][c], mul2(k[i], v2));
                    acc = fma2(q[i], S[i][c], acc);
                } else {
                    S[i][c] = fma2(k[i], v2, mul2(decay, S[i][c]));
                    acc = fma2(q[i], S[i][c], acc);
                }
            }
            float lo, hi;
            unpack2(acc, lo, hi);
            o[c] = lo + hi;
        }
    };

    float* out = p.out + (size_t)t0 * p.out_stride + (size_t)head * vdim + c0 + j0;
    int stage = 0;
#pragma unroll 1
    for (int left = t1 - t0; left > 0; left -= TB) {
        block_barrier(blockDim.x);
        const float* in = ring + stage * (TB * TOKEN);
        stage = stage + 1 == RING ? 0 : stage + 1;
        float o[TB * CC];
        if (left >= TB) {
#pragma unroll
            for (int tt = 0; tt < TB; ++tt) token(in + tt * TOKEN, o + tt * CC);
        } else {
#pragma unroll
            for (int tt = 0; tt < TB; ++tt) {
                if (tt < left) token(in + tt * TOKEN, o + tt * CC);
                else
#pragma unroll
                    for (int c = 0; c < CC; ++c) o[tt * CC + c] = 0.f;
            }
        }
        // sums over the LR lanes of the keys; lane r keeps the numbers r * KEEP .. (number n: token n / CC, column n % CC)
#pragma unroll
        for (int h = LR / 2; h >= 1; h >>= 1) {
            const bool up = (r & h) != 0;
#pragma unroll
            for (int i = 0; i < h * SH::KEEP; ++i) {
                const float give = up ? o[i] : o[i + h * SH::KEEP], keep = up ? o[i + h * SH::KEEP] : o[i];
                o[i] = keep + __shfl_xor_sync(0xffffffffu, give, h);
            }
        }
#pragma unroll
        for (int i = 0; i < SH::KEEP; ++i) {
            const int num = r * SH::KEEP + i, tt = num / CC, c = num % CC;
            if (tt < left && j0 + c < n_cols) {
                const float* tok = in + tt * TOKEN;
                out[(long long)tt * p.out_stride + c] =
                    WALK == PER_CHANNEL ? p.out_scale * o[i] : fmaf(CH ? tok[TOKEN - 4] : skip, tok[V + j0 + c], o[i]);
            }
        }
        out += TB * p.out_stride;
    }
#pragma unroll
    for (int c = 0; c < CC; ++c)
#pragma unroll
        for (int i = 0; i < RPV; ++i) {
            const int row = 4 * (r + LR * i);
            if (row < dim4 && j0 + c < n_cols) {
                float4 f;
                unpack2(S[2 * i][c], f.x, f.y); unpack2(S[2 * i + 1][c], f.z, f.w);
                *(float4*)(st + (size_t)(c0 + j0 + c) * dim4 + row) = f;
            }
        }
    pdl_launch_dependents();                              // (late: the next kernel's blocks would only sit and wait)
}

// ---- what a token brings besides q, k and v
// state space: scalars[t, h] = (exp(-exp(A_log[h]) dt), dt, -, -), dt = softplus(a[t, h] + dt_bias[h])
__global__ void __launch_bounds__(128) state_space_gates_kernel(const float* __restrict__ a, long long stride,
                                                                const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                                float* __restrict__ scalars, long long n, int heads) {
    pdl_wait();
    pdl_launch_dependents();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const long long t = i / heads;
    const int h = (int)(i % heads);
    const float z = a[t * stride + h] + dt_bias[h];
    const float dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
    *(float4*)(scalars + 4 * i) = make_float4(expf(-expf(a_log[h]) * dt), dt, 0.f, 0.f);
}

// decaying memory: w[t, h, i] = exp(-exp(z + w0)) in place, scalars[t, h, 0] = sum_i q_i u_i k_i.  One warp per (token, head).
__global__ void __launch_bounds__(128) memory_gates_kernel(float* __restrict__ w, long long w_stride, const float* __restrict__ w0,
                                                           const float* __restrict__ q, long long q_stride,
                                                           const float* __restrict__ k, long long k_stride,
                                                           const float* __restrict__ u, float* __restrict__ scalars, long long rows,
                                                           int heads, int dim) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const long long row = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (row >= rows) return;
    const long long t = row / heads;
    const int h = (int)(row % heads);
    float* wr = w + t * w_stride + (size_t)h * dim;
    const float* qr = q + t * q_stride + (size_t)h * dim;
    const float* kr = k + t * k_stride + (size_t)h * dim;
    float s = 0.f;
    for (int i = lane; i < dim; i += 32) {
        wr[i] = expf(-expf(wr[i] + w0[h * dim + i]));
        s = fmaf(qr[i] * u[h * dim + i], kr[i], s);
    }
    s = warp_sum(s);
    if (lane == 0) *(float4*)(scalars + 4 * row) = make_float4(s, 0.f, 0.f, 0.f);
}

// gated linear attention: w[t, c] = sigmoid(z)^(1/tau) with z = sum_r a[t, r] A_2[r, c] + b[c] for the channels c of all heads.
// A thread has one channel of DECAY_TOKENS tokens (8 in prompts, 1 in steps of few tokens); the sum runs over r in ascending order.
constexpr int DECAY_RANK = 64;                            // (the short vectors of a block's tokens pass through in pieces)
template <int DECAY_TOKENS>
__global__ void __launch_bounds__(128) channel_decays_kernel(const float* __restrict__ a, long long a_stride, const float* __restrict__ a2,
                                                             const float* __restrict__ b, float* __restrict__ w, long long w_stride,
                                                             int n_tokens, int n, int rank, float inv_tau) {
    __shared__ float a_s[DECAY_TOKENS][DECAY_RANK];
    pdl_wait();
    pdl_launch_dependents();
    const int c = blockIdx.x * 128 + threadIdx.x, t0 = blockIdx.y * DECAY_TOKENS, nt = min(DECAY_TOKENS, n_tokens - t0);
    float z[DECAY_TOKENS];
#pragma unroll
    for (int t = 0; t < DECAY_TOKENS; ++t) z[t] = 0.f;
    for (int r0 = 0; r0 < rank; r0 += DECAY_RANK) {
        const int nr = min(DECAY_RANK, rank - r0);
        if (r0 > 0) __syncthreads();
        for (int e = threadIdx.x; e < DECAY_TOKENS * nr; e += 128) {
            const int t = e / nr, r = e % nr;
            a_s[t][r] = t < nt ? a[(long long)(t0 + t) * a_stride + r0 + r] : 0.f;
        }
        __syncthreads();
        if (c < n) {
#pragma unroll 16
            for (int r = 0; r < nr; ++r) {
                const float v = a2[(size_t)(r0 + r) * n + c];
#pragma unroll
                for (int t = 0; t < DECAY_TOKENS; ++t) z[t] = fmaf(a_s[t][r], v, z[t]);
            }
        }
    }
    if (c >= n) return;
    const float bias = b[c];
#pragma unroll
    for (int t = 0; t < DECAY_TOKENS; ++t) {
        if (t >= nt) break;
        const float y = z[t] + bias;                      // log sigmoid(y) = -(max(-y, 0) + log(1 + e^-|y|))
        w[(long long)(t0 + t) * w_stride + c] = expf(-inv_tau * (fmaxf(-y, 0.f) + log1pf(expf(-fabsf(y)))));
    }
}

template <int LR, int RPV, int CC, int TB, int WALK>
int launch_scan(const ScanParams& p, int wide, cudaStream_t st) {
    using SH = Shape<LR, RPV, CC, TB, WALK>;
    // four walking warps a block, fewer where a step has so few (segment, head) pairs that more and smaller blocks spread better
    int warps = MAX_WARPS;
    while (warps > 1 && ((long long)((p.vdim + SH::WC * warps - 1) / (SH::WC * warps)) * p.heads * p.n_segments < 148 ||
                         SH::WC * (warps / 2) >= p.vdim)) warps /= 2;
    const size_t bytes = (size_t)RING * TB * SH::TOKEN * sizeof(float);
    auto kernel = scan_kernel<LR, RPV, CC, TB, WALK>;
    if (bytes > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
        return SPITE_LAUNCH_FAILED;
    dim3 grid((p.vdim + SH::WC * warps - 1) / (SH::WC * warps), p.heads, p.n_segments);
    // A step of single tokens is launched as a programmatic dependent; a longer walk in the ordinary way: started early, its
    // blocks would take the multiprocessors that the kernel before frees first, several to one, for the whole walk.
    if (p.n_tokens == p.n_segments) SPITE_LAUNCH(kernel, grid, 32 * (warps + 1), bytes, st, p, wide);
    else kernel<<<grid, 32 * (warps + 1), bytes, st>>>(p, wide);
    return spite_launch_status();
}

template <int WALK>
int choose_scan(const ScanParams& p, cudaStream_t st) {
    constexpr bool CH = WALK != PER_HEAD;
    const auto al = [](const void* x) { return ((uintptr_t)x & 15) == 0; };
    const int wide = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.q_stride % 4 == 0 && p.k_stride % 4 == 0 && p.v_stride % 4 == 0 &&
                     al(p.q) && al(p.k) && al(p.v) && (WALK == PER_CHANNEL || al(p.scalars)) && (!CH || (p.w_stride % 4 == 0 && al(p.w)));
    if (p.dim <= 32) return launch_scan<8, 1, 2, 8, WALK>(p, wide, st);
    if (p.dim <= 64) return launch_scan<8, 2, 2, 8, WALK>(p, wide, st);
    if (p.dim <= 128) return launch_scan<8, 4, 2, 8, WALK>(p, wide, st);
    if (p.dim <= 256) return launch_scan<16, 4, 2, 8, WALK>(p, wide, st);
    return launch_scan<32, 4, 4, 8, WALK>(p, wide, st);
}

int check_scan(const ScanParams* p) {
    if (!p || !p->q || !p->k || !p->v || !p->out || !p->state || !p->cu_seqlens || !p->slots) return SPITE_BAD_ARG;
    if (p->n_segments < 0 || p->n_tokens < 0 || p->heads < 1 || p->kv_heads < 1 || p->heads % p->kv_heads || p->dim < 1 || p->vdim < 1)
        return SPITE_BAD_ARG;
    const long long dim4 = (p->dim + 3) & ~3;
    if (p->slot_stride < (long long)p->heads * p->vdim * dim4 || p->out_stride < (long long)p->heads * p->vdim) return SPITE_BAD_ARG;
    if (p->q_stride < 1 || p->k_stride < 1 || p->v_stride < 1) return SPITE_BAD_ARG;
    if (p->slot_stride % 4 || ((uintptr_t)p->state & 15)) return SPITE_UNSUPPORTED;      // the state moves in 16-byte groups
    if (p->dim > 512 || p->heads > 65535 || p->n_segments > 65535) return SPITE_UNSUPPORTED;
    return SPITE_OK;
}

}  // namespace

// `a` [tokens, heads] with rows of a_stride: the projection's step columns; p->scalars is filled here
SPITE_API int spite_state_space_scan(const ScanParams* p, const float* a, long long a_stride, const float* a_log,
                                     const float* dt_bias, void* stream) {
    const int chk = check_scan(p);
    if (chk != SPITE_OK) return chk;
    if (!a || !a_log || !dt_bias || !p->scalars || p->w || a_stride < p->heads) return SPITE_BAD_ARG;
    if (p->n_segments == 0 || p->n_tokens == 0) return SPITE_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const long long n = (long long)p->n_tokens * p->heads;
    SPITE_LAUNCH(state_space_gates_kernel, (int)((n + 127) / 128), 128, 0, st, a, a_stride, a_log, dt_bias, (float*)p->scalars, n, p->heads);
    if (cudaGetLastError() != cudaSuccess) return SPITE_LAUNCH_FAILED;
    return choose_scan<PER_HEAD>(*p, st);
}

// p->w holds the decay's pre-activations on entry and the decays afterwards; `u` and `w0` [heads * dim]
SPITE_API int spite_decay_scan(const ScanParams* p, const float* w0, const float* u, void* stream) {
    const int chk = check_scan(p);
    if (chk != SPITE_OK) return chk;
    if (!w0 || !u || !p->scalars || !p->w || p->w_stride < (long long)p->heads * p->dim || p->kv_heads != p->heads || p->skip) return SPITE_BAD_ARG;
    if (p->n_segments == 0 || p->n_tokens == 0) return SPITE_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const long long rows = (long long)p->n_tokens * p->heads;
    if ((rows + 3) / 4 > 0x7fffffffLL) return SPITE_UNSUPPORTED;
    SPITE_LAUNCH(memory_gates_kernel, (int)((rows + 3) / 4), 128, 0, st, (float*)p->w, p->w_stride, w0, p->q, p->q_stride, p->k,
                 p->k_stride, u, (float*)p->scalars, rows, p->heads, p->dim);
    if (cudaGetLastError() != cudaSuccess) return SPITE_LAUNCH_FAILED;
    return choose_scan<PER_CHANNEL_BONUS>(*p, st);
}

// p->w [tokens, heads * dim] receives the decays, from the short vectors `a` [tokens, rank] (rows of a_stride), `a2` [rank,
// heads * dim] and `b` [heads * dim]
SPITE_API int spite_gated_linear_scan(const ScanParams* p, const float* a, long long a_stride, const float* a2, const float* b,
                                      int rank, float tau, void* stream) {
    const int chk = check_scan(p);
    if (chk != SPITE_OK) return chk;
    if (!a || !a2 || !b || rank < 1 || a_stride < rank || !(tau > 0.f) || !(p->out_scale == p->out_scale)) return SPITE_BAD_ARG;
    if (!p->w || p->w_stride < (long long)p->heads * p->dim || p->kv_heads != p->heads || p->skip) return SPITE_BAD_ARG;
    if (p->n_segments == 0 || p->n_tokens == 0) return SPITE_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const int n = p->heads * p->dim;
    const bool few = p->n_tokens <= 64;
    dim3 grid((n + 127) / 128, few ? p->n_tokens : (p->n_tokens + 7) / 8);
    if (grid.y > 65535) return SPITE_UNSUPPORTED;
    auto decays = few ? channel_decays_kernel<1> : channel_decays_kernel<8>;
    SPITE_LAUNCH(decays, grid, 128, 0, st, a, a_stride, a2, b, (float*)p->w, p->w_stride, p->n_tokens, n, rank, 1.f / tau);
    if (cudaGetLastError() != cudaSuccess) return SPITE_LAUNCH_FAILED;
    return choose_scan<PER_CHANNEL>(*p, st);
}
