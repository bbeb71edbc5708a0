// Argument blocks of the attention kernels.
#pragma once
#include "common.cuh"

#define SPITE_WINDOW_FULL 0      // keys 0..pos
#define SPITE_WINDOW_CHUNK 1     // keys of the query's chunk: floor(pos/size)*size .. pos
#define SPITE_WINDOW_SLIDING 2   // the last `size` keys: max(0, pos-size+1) .. pos

// The tokens of one step, flattened.  Token t belongs to segment seg_of_token[t]
// (one segment per request in the step) and sits at absolute position positions[t].
// block_table[seg * table_width + p / page_size] is the page that holds position p.
struct StepTokens {
    const int* positions;
    const int* seg_of_token;
    const int* block_table;
    int table_width;
    int n_tokens;
};

// One cache: keys at kv, values at kv + v_offset (elements); a page holds, for every
// kv head, page_size rows of head_dim elements: [pages][kv heads][page_size][head_dim].
// v_offset 0: the cache has keys only and a position's value is its key row.
// key_scale, if given, holds a factor per cached key, [pages][kv heads][page_size]: the score of a key is the product with its row
// times its factor (a norm of the keys whose rows are kept as projected, because they are the values too).
struct PagedCache {
    void* kv;
    long long v_offset;
    int n_pages;
    int page_size;
    int num_kv_heads;
    int head_dim;
    float* key_scale;
};

#define SPITE_PAIR_NEIGHBOURS 0   // pair i of a head is elements (2i, 2i+1)
#define SPITE_PAIR_HALVES 1       // pair i is elements (i, i + rotary_dim/2)

struct QkPrepareParams {
    const void* qkv;            // [tokens, (nq + 2 nkv) * head_dim]: q heads, k heads, v heads
    void* q_out;                // [tokens, nq * head_dim]
    const float* inv_freq;      // [rotary_dim / 2] rotation frequencies, or null: no rotation
    const float* q_gain;        // [head_dim] gain of the norm of q heads, or null (weightless)
    const float* k_gain;        // [head_dim] the same for k heads
    float qk_norm_eps;          // > 0: RMS norm of every q and k head
    int norm_before_rotation;   // the norm runs before the rotation instead of after it
    int pairing;                // SPITE_PAIR_*
    int rotary_dim;             // the first rotary_dim elements of a head rotate (even, <= head_dim)
    int temperature_floor;      // > 0: q *= ln(floor((pos+1)/floor) + 1) * temperature_scale + 1
    float temperature_scale;
    int num_heads;
    int write_cache;            // append k and v to the cache
    long long qkv_stride;       // elements between two tokens' rows of qkv (>= (nq + 2 nkv) * head_dim; 0: exactly that)
    float rot_amplitude;        // cos and sin of the rotation are multiplied by this (1, or 0 for unset: a pure rotation)
    // value blending: element i < v_mix_dim of kv head g's value becomes (1 - v_mix) v + v_mix * v_other[t * v_other_stride +
    // g * v_other_head + i] before it is cached (v_other null: no blending)
    const void* v_other;
    long long v_other_stride;
    int v_other_head;
    int v_mix_dim;
    float v_mix;
    // gates_out[t * nq + h] = sigmoid(qkv[t * qkv_stride + (nq + 2 nkv) * head_dim + h]) (null: no gate columns)
    float* gates_out;
    // bias[column] (float32, the columns of a token's row of qkv up to the last head's) is added to the projection's
    // output before anything else happens to it (null: none)
    const float* bias;
    int q_only;                 // the rows of qkv hold the q heads alone: this layer reads keys and values that another layer cached
    int norm_dim;               // > 0: a q or k head has this many elements (the rest of its head_dim are padding zeros): the
                                // per-head norm's mean is taken over them (0: over head_dim)
    // rotated values: element i < v_rotary_dim / 2 of a value head pairs with its partner by v_pairing (SPITE_PAIR_*) and the
    // pair turns by position * v_inv_freq[i] before it is cached (null: values are cached as they are)
    const float* v_inv_freq;
    int v_rotary_dim;
    int v_pairing;
    // what inv_freq and v_inv_freq lost when they were rounded to float32 (null: the angle is the rounded product)
    const float* inv_freq_low;
    const float* v_inv_freq_low;
    // the values are the projected keys (bias included): a row of qkv holds q heads and k heads alone, a cache of one plane
    // takes the keys as projected, and what the norm would multiply a key by goes to the cache's key_scale
    int values_are_keys;
};

// cos and sin of pos * (freq + low).  With `low` the product's own rounding error and the frequency's are put back to second
// order, so that the angle of a far position is as exact as that of a near one; without it the float32 product counts.
__device__ __forceinline__ void turn_of(float pos, const float* freq, const float* low, int i, float& c, float& s) {
    const float f = freq[i], a = pos * f;
    sincosf(a, &s, &c);
    if (low) {
        const float e = fmaf(pos, f, -a) + pos * low[i];      // (up to a few thousandths of a turn at position 100,000)
        const float c0 = c, k = 1.0f - 0.5f * e * e;
        c = fmaf(-e, s, c * k);
        s = fmaf(e, c0, s * k);
    }
}

struct AttentionParams {
    const void* q;              // [tokens, nq * head_dim]
    void* out;                  // [tokens, nq * head_dim]
    int num_heads;
    int window_kind;
    int window_size;
    float softmax_scale;
    int has_sink;               // the softmax's denominator also holds exp(sink_logit): a key every query sees
    float sink_logit;           // and that adds nothing to the output (a score of 0 puts exp(0) = 1 into the sum)
    const float* head_sinks;    // [num_heads] or null: with has_sink, head h's sink has the score head_sinks[h] instead
    const float* head_slopes;   // [num_heads] or null: head_slopes[h] * (query position - key position) is taken off a score
    const float* head_gates;    // [tokens, num_heads] or null: head h's output of token t is multiplied by head_gates[t * nq + h]
    int out_by_head_tokens;     // 0: out is [tokens, num_heads, head_dim]; n > 0: out is [num_heads, n, head_dim], head by head
                                // (n the tokens of the step), the order in which a product per head reads its rows
    float score_softcap;        // > 0: a scaled score s becomes cap * tanh(s / cap) before bias, mask and softmax
    // A number per head and distance (or null): head h's score of a key n positions before the query gets
    // distance_bias[h * (distance_len + 2 * SPITE_DISTANCE_PAD) + SPITE_DISTANCE_PAD + min(n, distance_len - 1)].  A row's ends
    // are repeated SPITE_DISTANCE_PAD times on either side, so that a tile of keys around them reads without a test per key.
    const float* distance_bias;
    const int* distance_runs;   // [distance_len] the smallest distance from which up to this one every head's number stays the same
    int distance_len;
};

#define SPITE_DISTANCE_PAD 64

// The numbers of head `head` by distance (null without a table).
__device__ __forceinline__ const float* distance_row_of(const AttentionParams& p, int head) {
    return p.distance_bias ? p.distance_bias + (size_t)head * (p.distance_len + 2 * SPITE_DISTANCE_PAD) + SPITE_DISTANCE_PAD : nullptr;
}

// Where the output row of (token, head) starts, in rows of head_dim elements.
__device__ __forceinline__ size_t out_row_of(const AttentionParams& p, int token, int head) {
    return p.out_by_head_tokens > 0 ? (size_t)head * p.out_by_head_tokens + token : (size_t)token * p.num_heads + head;
}

// The score of head `head`'s sink (only meaningful with has_sink).
__device__ __forceinline__ float sink_of(const AttentionParams& p, int head) {
    return p.head_sinks ? p.head_sinks[head] : p.sink_logit;
}
// What is taken off the score of a key `distance` positions before the query.
__device__ __forceinline__ float slope_of(const AttentionParams& p, int head) {
    return p.head_slopes ? p.head_slopes[head] : 0.f;
}
// A scaled score squashed into (-cap, cap), or itself without a cap.
__device__ __forceinline__ float capped(const AttentionParams& p, float s) {
    return p.score_softcap > 0.f ? p.score_softcap * tanhf(s / p.score_softcap) : s;
}
// The same for the tensor-core kernels, without a division or a call: with t = s / cap, s (1 - t^2/3 + 2 t^4/15 - ...), the
// Taylor series of the hyperbolic tangent to t^11, where |t| <= CAP_SERIES (what is left out is below 1e-7 of the result), and
// cap (1 - 2 / (e^(2t) + 1)) beyond, whose absolute error is a few float32 roundings of the cap.
#define CAP_SERIES 0.4f
#define CAP_C1 (-1.f / 3.f)
#define CAP_C2 (2.f / 15.f)
#define CAP_C3 (-17.f / 315.f)
#define CAP_C4 (62.f / 2835.f)
#define CAP_C5 (-1382.f / 155925.f)
__device__ __forceinline__ float reciprocal_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float capped_series(float s, float cap, float inv_cap) {
    const float t = s * inv_cap, y = t * t;
    float r = s * fmaf(y, fmaf(y, fmaf(y, fmaf(y, fmaf(y, CAP_C5, CAP_C4), CAP_C3), CAP_C2), CAP_C1), 1.f);
    if (fabsf(t) > CAP_SERIES)
        r = fmaf(-2.f * cap, reciprocal_approx(exp2_approx(t * 2.8853900817779268f) + 1.f), cap);      // (e^(2t) = 2^(2t / ln 2))
    return r;
}
// The tensor-core kernels are compiled in three forms: scores as they are, capped, and with everything else (a factor per key,
// a number per distance, a cap or none) chosen at run time.  With the choice of the cap made per score at run time, the decode
// kernel took a tenth longer without any cap.
enum ScoreForm { FORM_PLAIN = 0, FORM_CAP = 1, FORM_ANY = 2 };
static inline int score_form_of(const AttentionParams& p, const PagedCache& c) {
    return p.distance_bias || c.key_scale ? FORM_ANY : p.score_softcap > 0.f ? FORM_CAP : FORM_PLAIN;
}
static inline bool distance_bias_ok(const AttentionParams* p) {
    return !p->distance_bias || (p->distance_runs && p->distance_len >= 1 && p->distance_len <= (1 << 24));
}
// The score of a visible key n positions before the query, from the product `s` scaled by the softmax's scale; `key` is the
// key's own factor (1 without one), `inv_cap` 1 / score_softcap (0 without a cap), `number` what the distance adds.
template <int FORM>
__device__ __forceinline__ float score_of(const AttentionParams& p, float s, float key, float inv_cap, float slope, float number, int n) {
    if constexpr (FORM == FORM_PLAIN) return s - slope * (float)n;
    else {
        if constexpr (FORM == FORM_ANY) s *= key;
        if (FORM == FORM_CAP || inv_cap > 0.f) s = capped_series(s, p.score_softcap, inv_cap);
        s -= slope * (float)n;
        return FORM == FORM_ANY ? s + number : s;
    }
}
__device__ __forceinline__ float inverse_cap(const AttentionParams& p) { return p.score_softcap > 0.f ? 1.f / p.score_softcap : 0.f; }
// What the distance n (of either sign; a key behind the query is masked anyway) adds to a score.
__device__ __forceinline__ float number_at(const AttentionParams& p, const float* row, int n) {
    return row ? row[min(max(n, 0), p.distance_len - 1)] : 0.f;
}
// The factor of the first key of a tile that lies in one page (null without factors).
__device__ __forceinline__ const float* key_scale_of(const PagedCache& c, int page, int kvh, int position) {
    return c.key_scale ? c.key_scale + ((size_t)page * c.num_kv_heads + kvh) * c.page_size + position % c.page_size : nullptr;
}
// The factor on a finished output row.
__device__ __forceinline__ float gate_of(const AttentionParams& p, int token, int head) {
    return p.head_gates ? p.head_gates[(size_t)token * p.num_heads + head] : 1.f;
}

// The sink folded into a finished softmax state: `m` and `l` are the maximum and the sum of exp(s - m) over the
// real keys (natural-log units).  Afterwards l is the whole denominator relative to max(m, sink); the return
// value is the factor by which the accumulated values shrink to the same reference.
__device__ __forceinline__ float fold_sink(const AttentionParams& p, int head, float m, float& l) {
    if (!p.has_sink) return 1.f;
    const float sink = sink_of(p, head);
    const float m2 = fmaxf(m, sink);
    const float f = (m == -INFINITY) ? 0.f : expf(m - m2);
    l = l * f + expf(sink - m2);
    return f;
}

// What the tensor-core attention kernels need beyond the above.  Two kernels share a step:
// segments of few tokens (decode) go to the one that splits the keys among blocks, segments
// of many tokens (prompt portions) to the one that gives every warp its own rows; each kernel
// serves the segments whose token count lies in [seg_min_tokens, seg_max_tokens].
struct AttnMmaExtra {
    const int* cu_seqlens;       // [segments + 1]
    float* o_part;               // [tokens, heads, splits, head_dim]   (splits > 1)
    float* ml_part;              // [tokens, heads, splits, 2]          running maximum, sum
    int n_segments;
    int tokens_per_block;        // tokens whose (token, head) rows fill one block
    int n_splits;
    int seg_min_tokens;
    int seg_max_tokens;
};

// The same for the decode kernel whose last-arriving block merges the key splits itself.
struct AttnDecodeExtra {
    const int* cu_seqlens;       // [segments + 1]
    float* partial;              // [blocks, kv heads, splits, 16, head_dim + 4]   (splits > 1)
    int* tickets;                // [blocks, kv heads], zero between launches      (splits > 1)
    int n_segments;
    int tokens_per_block;
    int n_splits;
    int seg_min_tokens;
    int seg_max_tokens;
    int cache_settled;           // the cache rows of positions before each request's first token of this step were
                                 // written at least two launches ago on this stream: they may be read before the wait
};

__device__ __forceinline__ int window_lowest(int kind, int size, int pos) {
    if (kind == SPITE_WINDOW_CHUNK) return (pos / size) * size;
    if (kind == SPITE_WINDOW_SLIDING) return max(0, pos - size + 1);
    return 0;
}
