"""The contract between the layer parts and the kernels.

A `KernelSet` is bound to one activation type (bfloat16 or float32).  The
residual stream, norm gains, router weights, softmax statistics and logits are
float32 in both sets.  Parts call these methods and nothing else to touch the
device; a kernel set never learns which model or layer it serves.

Shapes use M for the tokens of the step, d for the model width, T for the
activation type.  All tensors are contiguous and live on the set's device.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


class KernelError(RuntimeError):
    """A kernel refused its arguments or could not be launched."""


class KernelTimeout(KernelError):
    """A kernel gave up a bounded wait and left its output incomplete: the results of the steps
    since the last check cannot be trusted (ExecutorError in crates/spite-executor/src/lib.rs:88-100
    is the counterpart: a typed error instead of wrong logits)."""


@dataclass
class Routing:
    """Result of `moe_route` for M tokens, E experts and k choices per token."""
    expert_ids: torch.Tensor     # [k, M] int32
    weights: torch.Tensor        # [k, M] float32, sigmoid of the chosen logits
    offsets: torch.Tensor        # [k, E + 1] int32: places of each expert's tokens in sorted_rows
    sorted_rows: torch.Tensor    # [k, M] int32: token indices ordered by expert, ascending within one
    logits: Optional[torch.Tensor] = None   # [M, E] float32 if asked for
    sorted_weights: Optional[torch.Tensor] = None   # [k, M] float32: weights[slot][sorted_rows[slot][i]] at place i


@dataclass(frozen=True)
class DistanceBias:
    """A number per head and distance for attention scores: head h's score of a key n positions before the query gets
    padded[h, PAD + min(n, length - 1)].  The rows' ends are repeated PAD times on either side (a kernel reads whole tiles of
    keys around them); `runs`[n] is the smallest distance from which up to n every head's number stays the same."""
    PAD = 64
    padded: torch.Tensor         # float32 [heads, PAD + length + PAD]
    runs: torch.Tensor           # int32 [length]

    @property
    def length(self) -> int:
        return self.runs.numel()

    @classmethod
    def from_rows(cls, table: torch.Tensor, row_of: list) -> "DistanceBias":
        """`table` [rows, heads]: row row_of[n] serves distance n, the last entry every distance from there on."""
        dev = table.device
        index = torch.tensor([row_of[0]] * cls.PAD + list(row_of) + [row_of[-1]] * cls.PAD, dtype=torch.long, device=dev)
        runs, start = [], 0
        for n, row in enumerate(row_of):
            if n and row != row_of[n - 1]:
                start = n
            runs.append(start)
        return cls(table.to(torch.float32)[index].t().contiguous(), torch.tensor(runs, dtype=torch.int32, device=dev))


class KernelSet:
    """Interface; see `CudaKernels` for the product implementation."""

    dtype: torch.dtype
    device: torch.device

    def errors(self) -> dict:
        """{kernel library: code} for every library one of whose kernels gave up a bounded wait since
        the last call; reading clears.  Does not wait for the device: call it after a point at
        which the host has waited for the step's results."""
        return {}

    # ---- elementwise
    def embed(self, table, token_ids, out_h, *, scale=1.0, position_table=None, positions=None, copies=1):
        """out_h[m, :] (float32) = table[token_ids[m], :] (T) * scale; with `copies` n, out_h is [M, n, d] and every row is
        written n times (the start of several residual streams); with a `position_table` [P, d] (T)
        and `positions` [M] int32, + position_table[positions[m], :] (the factor applies to the token's row only)."""
        raise NotImplementedError

    def pack_pair(self, a, b, out, *, refill=None):
        """out[m, :] (T) = [a[m, :]; b[m, :]] for two float32 streams [M, d]; with `refill` [d] float32 every
        row of `a` becomes that vector afterwards (the stream is restarted for a product that adds into it)."""
        raise NotImplementedError

    def transform_logits(self, logits, *, scale=1.0, softcap=None):
        """In place: logits *= scale; then, with a cap, logits = cap * tanh(logits / cap)."""
        raise NotImplementedError

    def rms_norm(self, h, gain, eps, out, rows=None):
        """out[i, :] (T or float32) = h[r] * rsqrt(mean(h[r]^2) + eps) * gain, r = rows[i] if rows else i.
        h float32 [*, d], gain float32 [d]."""
        raise NotImplementedError

    def rms_norm_residual(self, y, gain, eps, mult, h, *, next_gain=None, next_out=None):
        """A sublayer's output is normed before it joins the residual stream:
        h[m, :] += mult * y[m, :] * rsqrt(mean(y[m]^2) + eps) * gain (y, h float32 [M, d]); with `next_out` [M, d]
        (T) also the norm the next sublayer reads, of the row just made: next_out = h * rsqrt(mean(h^2) + eps) * next_gain;
        `next_out` without `next_gain`: the row itself in next_out's type (the next sublayer reads the stream unnormed)."""
        raise NotImplementedError

    def cast_rows(self, h, out):
        """out (T) = h (float32), element by element: what a sublayer without a norm in front of it reads."""
        raise NotImplementedError

    def short_conv(self, x, w, out, batch, state, *, channels, activation=None, state_offset=0, bias=None):
        """A short causal convolution over time on the first `channels` columns of a projection's float32 output x
        [M, >= channels + c]: out[t, ch] = act(sum_j w[ch, j] * x[t - taps + 1 + j, ch]) within each segment, w float32
        [channels, taps]; rows before a segment's first token come from the request's slot, state[slot, state_offset :
        state_offset + (taps - 1) * channels] (float32 [taps - 1, channels], oldest first; zeros at the start of a
        sequence), which then receives the sequence's last taps - 1 rows of x.  The c = out.shape[1] - channels columns behind
        the channels are passed on unchanged.  out [M, channels + c] is T or float32; `activation` None or "silu".
        `bias` float32 [channels] is added to a channel's sum before the activation.
        With one tap nothing is carried and `state` may be None."""
        raise NotImplementedError

    def fill_rows(self, out, vec, *, accumulate=False, other=None):
        """out[m, :] (float32 [M, d]) = vec (float32 [d]), or += vec: a bias laid down for a product that adds to it.  `other`
        (float32 [M, d]) is added row by row ahead of the vector."""
        raise NotImplementedError

    def head_norm_gate(self, x, out, *, heads, size, gates=None, gate_column=0, gain=None, eps=None, gate_activation="sigmoid",
                       out_column=None):
        """What stands between a mixer's heads and its output projection.  x [M, heads * size] (T, or float32: the
        result of a recurrence), out [M, heads * size] (T; may be x):
        out[m, h, j] = x[m, h, j] * r * gain[h * size + j] * sigmoid(gates[m, gate_column + h * size + j]) with
        r = rsqrt(mean_j x[m, h, :]^2 + eps) if `eps` is given (a norm of every head without a gain of its own), else 1;
        `gates` (a 2-D tensor of x's type, the gate columns of a wider product) and `gain` (float32) may be left out; a gain
        of `size` elements is shared by the heads.
        `gate_activation` "silu": the factor is z * sigmoid(z) of the gate column z instead of sigmoid(z).
        `out_column` c: out is a wider 2-D tensor and the result goes into its columns from c on."""
        raise NotImplementedError

    def turn_heads(self, x, out, batch, *, heads, size, rotation=None, scale=1.0, out_column=0):
        """The other way from a mixer's heads to its output projection, for heads whose values were cached rotated by their
        own position: out[m, out_column + h * size + e] (T, a 2-D tensor) = scale * (x[m, h, :size] turned back)[e], every pair
        of `rotation` by minus the angle that the token's position turns it by (None: not turned).  x [M, heads * head_dim]
        (T) with head_dim >= size: what lies behind a head's first `size` elements is left out."""
        raise NotImplementedError

    def gate_group_norm(self, x, z, gain, out, *, groups, eps, z_column=0):
        """A gate first, a norm behind it: v = x[m, :] * silu(z[m, z_column:]); out[m, e] (T) = v[e] / sqrt(mean of v^2 over e's
        part + eps) * gain[e], `groups` equal parts; x float32 [M, n], z float32 [M, >= z_column + n], gain float32 [n]."""
        raise NotImplementedError

    def token_shift(self, x, mu, out, batch, state, *, state_offset=0, offsets_out=None):
        """out[g, m, :] (T) = x[m, :] + (x'[m, :] - x[m, :]) * mu[g, :] with x' the row of the token before in the sequence: for
        a segment's first token the row in its request's slot (float32, state[slot, state_offset : state_offset + d]; zeros
        at the start of a sequence), which then receives the segment's last row.  x [M, d] (T), mu float32 [n, d], out
        [n, M, d]; `offsets_out` (int32 [n + 1]) receives g * M: the groups of a `batched_linear` over out."""
        raise NotImplementedError

    # ---- several residual streams
    def streams(self, x, *, y=None, bias=None, scale=None, mix=None, w_out=None, w_in=None, gain=None, eps=None, next_out=None,
                rows=None, write_back=True):
        """Everything between two sublayers of a model with n residual streams x float32 [M, n, d] (hyper-connections).
        With the sublayer's output y float32 [M, d]: v = (y + bias) * scale, and all streams at once from the old ones
        x_t <- sum_s mix[s, t] x_s + w_out[t] v (mix [n, n], [from, to]).  With `next_out` [rows, d] (T or float32): what the
        next sublayer reads, u = sum_s w_in[s] x_s of the streams just made, next_out = u / sqrt(mean(u^2) + eps) * gain (u
        itself without a gain).  `rows` int32: only these tokens (row i of next_out is token rows[i]); `write_back` False:
        the new streams are used for u and not stored.  All coefficients float32."""
        raise NotImplementedError

    # ---- matrix products: y = x W^T with W [out, in]
    def linear(self, x, w, out, *, accumulate=False, row_scale=None, activation=None, bias=None, act_params=None):
        """out[M, N] = x[M, K] @ w[N, K]^T.  `out` is T, or float32 (logits); with
        `accumulate` it is float32 and the product is added to it (residual stream).
        `row_scale` [M] float32 multiplies the product's rows.  `activation` (with an output of type T):
        "relu2": out = relu(s y)^2; "gelu_tanh": out = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), z = s y; "tanh";
        "xielu" with `act_params` (a, b): a z^2 + z / 2 for z > 0, else b (e^z - 1 - z) + z / 2.  `bias` float32 [N] (with an
        output of type T) is added to the scaled product before the activation: z = s y + bias."""
        raise NotImplementedError

    def batched_linear(self, x, w, offsets, out):
        """out[g, M, N] (float32) = x[g, M, K] @ w[g, N, K]^T: one product per group on rows of its own; offsets int32 [G + 1]
        on the device holds g * M."""
        raise NotImplementedError

    def linear_swiglu(self, x, w_gate_up, out, *, row_scale=None, activation="silu"):
        """out[M, F] (T) = silu(s g) * (s u) with g = x @ w[:F]^T, u = x @ w[F:]^T, s = row_scale or 1; `activation`
        "gelu_tanh": the gate's function is gelu in its tanh form (as in `linear`) instead of silu."""
        raise NotImplementedError

    def grouped_linear_swiglu(self, x, w_gate_up, sorted_rows, offsets, row_scale, out):
        """Row i of `out` [M, F] (sorted order) is the SwiGLU of token sorted_rows[i] through the
        expert whose range of `offsets` holds i; w_gate_up [E, 2F, K]; row_scale [M] by token."""
        raise NotImplementedError

    def grouped_linear_act(self, x, w_up, sorted_rows, offsets, row_scale, out, *, activation="relu2"):
        """Row i of `out` [M, F] (sorted order) is act(s * (x[sorted_rows[i]] @ w_up[e]^T)) for the expert e whose
        range of `offsets` holds i; w_up [E, F, K]; row_scale [M] by token; "relu2": act(y) = relu(y)^2."""
        raise NotImplementedError

    def grouped_linear_accumulate(self, a, w_down, sorted_rows, offsets, h, *, row_scale=None):
        """h[sorted_rows[i], :] (float32) += s_i * (a[i, :] @ w_down[expert of i]^T); w_down [E, d, F];
        `row_scale` [M] float32 by place i in the sorted order (s_i = 1 without it)."""
        raise NotImplementedError

    def grouped_linear_rows(self, a, w, rows, offsets, out, *, a_sorted=False):
        """out[rows[i], :N] (T) = a[rows[i], :K] @ w[g]^T for every place i of group g's range of `offsets`;
        a [R, lda >= K], w [G, N, K], out [R, ldc >= N].  Rows of `a` and `out` that no place names, and columns
        beyond K and N, are neither read nor written (a product per head: the rows are (token, head) pairs).
        With `a_sorted`, `a` lies in the list's order already: place i reads a[i, :K]."""
        raise NotImplementedError

    # ---- cache
    def clear_pages(self, kv, page_ids):
        """Zero the pages `page_ids` (a list of ints) of every cache of a group; `kv` is the group's tensor
        [caches, 2, pages, kv heads, page_size, head_dim].  The engine does this when it hands a page out,
        so that a request never multiplies a masked key's zero weight with what another request left there."""
        raise NotImplementedError

    # ---- attention
    def qk_prepare(self, qkv, q_out, batch, cache, *, num_heads, rotation, qk_norm, temperature,
                   value_mix=None, gates_out=None, bias=None, q_only=False, norm_dim=None, value_rotation=None,
                   values_are_keys=False):
        """Encode positions of q and k, normalise, scale q, append k and v to the cache.
        `bias` float32 [(nq + 2 nkv) hd]: added to the projection's columns before anything else.  `q_only`: a row of
        qkv holds the q heads alone (and `bias` theirs): the layer reads keys and values that another layer cached.
        qkv [M, >= (nq + 2 nkv) hd] T -> q_out [M, nq hd] T; `cache` is a `LayerCache`.
        `rotation`: a `parts.Rotation` or None; `qk_norm`: a `parts.QkNorm` or None (RMS norm of
        every q and k head, after the rotation unless it says before); `temperature`:
        (floor, scale) or None: q *= ln(floor((pos + 1) / floor) + 1) * scale + 1.
        `value_mix` = (other [M, *] T, column, head stride, value size, lam): element i < value size of kv head g's
        value becomes (1 - lam) v + lam * other[m, column + g * head stride + i] before it is cached.
        `gates_out` float32 [M, nq]: receives sigmoid(qkv[m, (nq + 2 nkv) hd + h]), the columns after the heads.
        `norm_dim`: a q or k head has this many elements and zeros behind them up to hd (a cache row wider than the key):
        the per-head norm takes its mean over them.
        `value_rotation`: a `parts.Rotation` over the leading elements of a value head: a value turns by its own position
        before it is cached.  `values_are_keys`: a row of qkv holds q and k heads alone ((nq + nkv) hd columns, `bias` too),
        and the value of a position is its key as projected, bias included; there is no rotation and no gain for k.  The cache has
        one plane, which takes the keys as projected, and a factor per key (`cache.key_scale` [pages, nkv, page_size]), which
        receives what the norm multiplies the key by (1 without a norm)."""
        raise NotImplementedError

    def paged_attention(self, q, out, batch, cache, *, num_heads, window, softmax_scale, cache_settled=False,
                        sink_logit=None, head_sinks=None, head_slopes=None, head_gates=None, out_by_head=False,
                        score_softcap=None, distance_bias=None):
        """out[M, nq hd] = softmax(q K^T * scale over the visible cached keys) V.
        `score_softcap` c: a scaled score s becomes c * tanh(s / c) before anything else happens to it.
        `out_by_head`: the result is laid out head by head instead, out[nq, M, hd] (the order in which a product per
        head reads its rows).
        `sink_logit`: the softmax's denominator also holds exp(sink_logit), a key without a value;
        `head_sinks` float32 [nq]: the same with a score of its own for every head.
        `head_slopes` float32 [nq]: slope_h * (query position - key position) is taken off head h's scores.
        `distance_bias`, a `DistanceBias`: a number per head and distance is added to a score (behind scale and cap).
        `head_gates` float32 [M, nq]: head h's output for token m is multiplied by head_gates[m, h].
        A cache with one plane (`cache.kv.shape[0] == 1`) holds keys only, and the value of a position is its key row.
        A cache with `key_scale` (float32 [pages, nkv, page_size]): the product with a key row is multiplied by the key's factor
        (ahead of scale and cap).
        `cache_settled`: the caller promises that the cache rows of positions before each request's first
        token of this step were written by earlier steps (not by the one or two kernels launched just
        before this call), so a kernel may fetch them while the kernel before still runs."""
        raise NotImplementedError

    # ---- attention through latents
    def latent_prepare(self, down, cq_out, batch, cache, *, q_rank, kv_rank, rotation, q_gain, kv_gain, eps,
                       num_gates=0, gates_out=None):
        """One row of `down` (float32 [M, >= q_rank + kv_rank + rot + num_gates]) holds a token's query latent, its
        key/value latent, the key part that all heads share and the gate columns.  cq_out [M, q_rank] (T) =
        RMS norm of the query latent * q_gain; the cache row of the token's position becomes [RMS norm of the
        key/value latent * kv_gain; the shared part rotated by `rotation` (either pairing, times its amplitude);
        zeros up to the row's size]; gates_out [M, num_gates] float32 = sigmoid of the gate columns."""
        raise NotImplementedError

    def latent_queries(self, q, q_out, batch, *, num_heads, head_dim, kv_rank, rotation, rows_out, offsets_out,
                       sorted_out=None):
        """q [M, nq (head_dim + rot)] (T): every head's last `rot` elements are rotated (as in `latent_prepare`) into
        q_out[m, h, kv_rank : kv_rank + rot], and q_out's elements behind them become zero (q_out [M, nq, row] T; its
        first kv_rank elements are left for the product that follows).  Also lists the (token, head) rows head by
        head: rows_out[h M + m] = m nq + h, offsets_out[h] = h M (int32 [nq M] and [nq + 1]); `sorted_out` [nq M, head_dim]
        (T), if given, receives the heads' unrotated parts in that order: sorted_out[h M + m] = q[m, h, :head_dim]."""
        raise NotImplementedError

    # ---- recurrent mixers
    def mlstm_scan(self, proj, out, batch, state, *, heads, dim, vdim, gate_cap, q_scale, columns, i_bias, f_bias,
                   chunked=None):
        """Matrix memory with exponential gates, token by token, for every segment of the step from the state its
        request's slot holds (all zeros: the start of a sequence); the slot receives the state after the segment's
        last token.  proj float32 [M, *] holds, from the columns `columns` = (q, k, v, i, f) on, q and k
        [heads * dim], v [heads * vdim] and the gates' pre-activations [heads]; out float32 [M, heads * vdim];
        state float32 [slots, heads, `mlstm_state_size(dim, vdim)`].
        i = cap tanh((a + i_bias) / cap), f = logsigmoid(cap tanh((c + f_bias) / cap)), m' = max(f + m, i),
        S' = exp(f + m - m') S + exp(i - m') k v^T, n' alike with k, out = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6),
        q times `q_scale`.  All float32.  `chunked`: walk the segments 32 tokens at a time (the same sums in another
        order) instead of token by token; None leaves the choice to the kernel set."""
        raise NotImplementedError

    @staticmethod
    def mlstm_state_size(dim: int, vdim: int) -> int:
        """Floats of one head's state: S [dim, vdim], then one copy of (n [dim], m) for every 32 value columns, each
        rounded up to a multiple of four floats."""
        return dim * vdim + -(-vdim // 32) * (-(-(dim + 1) // 4) * 4)

    def delta_scan(self, x, out, batch, state, *, heads, kv_heads, dim, vdim, columns, a_log, dt_bias, q_scale,
                   unit_eps=1e-6, state_offset=0, split_rows=None):
        """The gated delta rule, token by token, for every segment of the step from the matrix its request's slot holds
        (zeros: the start of a sequence); the slot receives the matrix after the segment's last token.  x float32 [M, *]
        holds, from the columns `columns` = (q, k, v, b, a) on, q and k [kv_heads * dim], v [heads * vdim] and two
        numbers a head; out float32 [M, heads * vdim]; state float32 [slots, *], head h's S [dim, vdim] row-major at
        state[slot, state_offset + h * dim * vdim].  Head h reads q/k head h // (heads / kv_heads).
        k <- k / sqrt(|k|^2 + unit_eps), q <- q / sqrt(|q|^2 + unit_eps) * q_scale, beta = sigmoid(b),
        g = exp(-exp(a_log[h]) * softplus(a + dt_bias[h])); S <- g S; u = beta (v - S^T k); S <- S + k u^T; out = S^T q.
        All float32.  `split_rows`: more lanes share a value column's key rows (the same sums in another order; for steps
        with long segments); None leaves the choice to the kernel set."""
        raise NotImplementedError

    @staticmethod
    def scan_state_size(dim: int, vdim: int) -> int:
        """Floats of one head's state in the two scans below: value column by value column, its keys padded to a multiple of four."""
        return vdim * (-(-dim // 4) * 4)

    def state_space_scan(self, q, k, v, step, out, batch, state, *, heads, kv_heads, dim, vdim, a_log, dt_bias, skip,
                         state_offset=0):
        """A state space with one decay per head and token (Mamba-2), for every segment of the step from the matrices its
        request's slot holds (zeros: the start of a sequence); the slot receives the matrices after the segment's last
        token.  Per head h: dt = softplus(step + dt_bias[h]); S <- exp(-exp(a_log[h]) dt) S + dt k v^T; out = S^T q + skip[h] v.
        q, k, v, step are pairs (float32 tensor [M, *], first column) of widths kv_heads * dim (twice), heads * vdim and heads;
        head h reads q and k of head h // (heads / kv_heads); out float32 [M, heads * vdim]; state float32 [slots, *], head h's
        S at state[slot, state_offset + h * scan_state_size(dim, vdim)], transposed ([vdim, keys]).  All float32."""
        raise NotImplementedError

    def decay_scan(self, r, k, v, w, out, batch, state, *, heads, dim, vdim, w0, u, state_offset=0):
        """A memory that decays per key channel (RWKV), walked and kept as above: out = S^T r + (sum_i r_i u_i k_i) v, then
        S <- diag(exp(-exp(w + w0))) S + k v^T.  w float32 [M, heads * dim] holds the decay's pre-activations and is
        overwritten with the decays; w0, u float32 [heads * dim]."""
        raise NotImplementedError

    def gated_linear_scan(self, q, k, v, a, w, out, batch, state, *, heads, dim, vdim, a2, a2_bias, tau, q_scale, state_offset=0):
        """Gated linear attention, walked and kept as above: S <- diag(w) S + k v^T, then out = q_scale S^T q, with the decays
        w = sigmoid(a A_2 + a2_bias)^(1 / tau) per head and key channel made first.  q, k, v and a (the short vectors of
        a2.shape[0] elements) are pairs (float32 tensor, first column); a2 float32 [rank, heads * dim] (input-major), a2_bias
        float32 [heads * dim]; w float32 [M, heads * dim] receives the decays."""
        raise NotImplementedError

    # ---- mixture of experts
    def moe_identity(self, x, routing, first_identity, out, *, accumulate=True):
        """Experts that return their input: out[m, :] (float32) (+)= sum over the choice slots s whose expert id
        routing.expert_ids[s, m] >= first_identity of routing.weights[s, m] * x[m, :] (x is T).  Without `accumulate`
        every row of out is written (zeros where no such expert was chosen)."""
        raise NotImplementedError

    def moe_route(self, x, w_router, top_k, want_logits=False, scoring="sigmoid", choice_bias=None, logit_bias=None) -> Routing:
        """Router logits in float32 (plus `logit_bias`, float32 [E], if given), the `top_k` largest per token (equal ones: the lower expert first), the
        tokens sorted by expert for every choice slot.  `scoring` "sigmoid": the weight of a choice is the sigmoid
        of its logit; "softmax_renorm": its share of the softmax over all experts, divided by the sum of the
        chosen shares (+ 1e-20); `sorted_weights` is filled for it.  "softmax_biased": the experts are ordered by their
        softmax share plus `choice_bias` (float32 [E]), and the weight of a choice is its share alone (not renormalised);
        `sorted_weights` is filled."""
        raise NotImplementedError

    # ---- sampling
    def argmax(self, logits):
        """[R] int32: index of the maximum of each row, the highest index among equals."""
        raise NotImplementedError

    def sample(self, logits, *, temperature, top_k, top_p, min_p, repetition_penalty,
               context, context_offsets, rng_state):
        """[R] int32 tokens; `rng_state` [R] int64 is advanced in place for rows that draw."""
        raise NotImplementedError
