"""Gated linear attention as a mixer.

Per head a matrix S [dim, vdim], zero at the start of a sequence, carried from token to token in float32 in the request's
state slot:

    q = W_q h * q_scale,  k = W_k h  (heads x dim),   v = W_v h,  gate = silu(W_g h)  (heads x vdim)
    w = sigmoid(W_a2 (W_a1 h) + b)^(1/tau)                                             per head and key channel
    S <- diag(w) S + k v^T;   o = S^T q
    out = W_o [ o_h / rms(o_h) * gain for every head, concatenated, * gate ]

One product makes q, k, v, the gate's columns and the short vector W_a1 h as float32 sums; `gated_linear_scan` turns the short
vectors into decays (the second small product, the bias, the sigmoid and the root in one kernel, float32 from end to end) and
walks every segment of the step; `head_norm_gate` norms the heads, applies gain and gate; the output projection adds into (or
fills) the stream.
"""
from __future__ import annotations

import torch

from ..cache import FixedState
from ..config.specs import ConfigError
from ..kernels.api import KernelSet
from .base import Mixer, ParamSpec, register_mixer


@register_mixer("gated_linear_attention")
class GatedLinearAttention(Mixer):
    graph_safe = True
    can_store = True
    kernel_libraries = ("gemm_simt", "scan")

    def __init__(self, ctx, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, decay_rank: int, tau: float,
                 norm_eps: float, q_scale: float | None = None):
        """`head_dim`: size of a head's q and k; `value_dim`: of its v and its output; `decay_rank`: rows of the first of the two
        matrices that make the decay; `tau`: the root taken of it; `norm_eps`: of the heads' norm, whose gain the heads share;
        `q_scale`: factor on q (default head_dim^-1/2)."""
        super().__init__(ctx)
        self.d, self.H, self.kd, self.vd = int(hidden_size), int(num_heads), int(head_dim), int(value_dim)
        self.rank = int(decay_rank)
        if min(self.d, self.H, self.kd, self.vd, self.rank) < 1:
            raise ConfigError("gated_linear_attention: sizes must be positive")
        if self.kd > 512:
            raise ConfigError(f"gated_linear_attention: head_dim {self.kd} exceeds the scan kernel's 512")
        if not float(tau) > 0 or not float(norm_eps) > 0:
            raise ConfigError("gated_linear_attention: tau and norm_eps must be positive")
        self.tau, self.eps = float(tau), float(norm_eps)
        self.q_scale = float(q_scale) if q_scale is not None else self.kd ** -0.5
        nk, nv = self.H * self.kd, self.H * self.vd
        self.nk, self.nv = nk, nv
        self.heads_size = nv
        # columns of the one product: q, k, v, the gate, the decay's short vector (then padding)
        self.k_column, self.v_column, self.gate_column, self.a_column = nk, 2 * nk, 2 * nk + nv, 2 * nk + 2 * nv
        self.n_columns = -(-(self.a_column + self.rank) // 8) * 8
        self.state_matrices = self.H * KernelSet.scan_state_size(self.kd, self.vd)
        self.w_in = self.w_out = self.a2 = self.a2_bias = self.gain = None
        self._scaled_gain = {}

    def param_specs(self):
        d, nk, nv = self.d, self.nk, self.nv
        return {"q_proj": ParamSpec((nk, d)), "k_proj": ParamSpec((nk, d)), "v_proj": ParamSpec((nv, d)), "gate_proj": ParamSpec((nv, d)),
                "decay_in": ParamSpec((self.rank, d)), "decay_out": ParamSpec((nk, self.rank)), "decay_bias": ParamSpec((nk,)),
                "norm": ParamSpec((self.vd,), "ones"), "o_proj": ParamSpec((d, nv))}

    def bind(self, params):
        dt, f32 = self.ctx.dtype, torch.float32
        rows = [params[n].to(dt) for n in ("q_proj", "k_proj", "v_proj", "gate_proj", "decay_in")]
        rows.append(torch.zeros((self.n_columns - self.a_column - self.rank, self.d), dtype=dt, device=rows[0].device))
        self.w_in = torch.cat(rows, 0).contiguous()
        self.w_out = params["o_proj"].to(dt).contiguous()
        self.a2 = params["decay_out"].to(f32).t().contiguous()           # input-major: neighbouring channels lie side by side
        self.a2_bias = params["decay_bias"].to(f32).contiguous()
        self.gain = params["norm"].to(f32).contiguous()
        self._scaled_gain = {1.0: self.gain}

    def gain_times(self, scale: float):
        """The gain with a factor on the whole mixer folded in (float32)."""
        if scale not in self._scaled_gain:
            self._scaled_gain[scale] = (self.gain * scale).contiguous()
        return self._scaled_gain[scale]

    def weight_bytes(self):
        n = self.w_in.numel() + (0 if self.w_out is None else self.w_out.numel())
        return n * self.w_in.element_size() + self.a2.numel() * 4

    def cache_request(self):
        return None, FixedState((self.state_matrices,), torch.float32)

    def heads(self, x, out, column, batch, cache, scale=1.0):
        k = self.k
        M, dev = x.shape[0], x.device
        proj = torch.empty((M, self.n_columns), dtype=torch.float32, device=dev)
        k.linear(x, self.w_in, proj)                              # float32 sums: nothing that enters the recurrence is rounded
        w = torch.empty((M, self.nk), dtype=torch.float32, device=dev)
        o = torch.empty((M, self.nv), dtype=torch.float32, device=dev)
        k.gated_linear_scan((proj, 0), (proj, self.k_column), (proj, self.v_column), (proj, self.a_column), w, o, batch, cache.state,
                            heads=self.H, dim=self.kd, vdim=self.vd, a2=self.a2, a2_bias=self.a2_bias, tau=self.tau,
                            q_scale=self.q_scale)
        k.head_norm_gate(o, out, heads=self.H, size=self.vd, gates=proj, gate_column=self.gate_column, gain=self.gain_times(scale),
                         eps=self.eps, gate_activation="silu", out_column=column)

    def forward(self, x, h, batch, cache, accumulate=True):
        a = torch.empty((x.shape[0], self.nv), dtype=x.dtype, device=x.device)
        self.heads(x, a, 0, batch, cache)
        self.k.linear(a, self.w_out, h, accumulate=accumulate)
