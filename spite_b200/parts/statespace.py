"""A selective state space with one decay per head (Mamba-2) as a mixer.

Per head a matrix S [state, vdim], zero at the start of a sequence, carried from token to token in float32 in the
request's state slot:

    [z | x | B | C | a] = W_in h                       (heads * vdim, heads * vdim, groups * state twice, heads)
    x, B, C <- silu(conv(x, B, C) + bias)              a causal convolution over time per channel
    dt = softplus(a + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x        (head h reads B and C of group h // (heads / groups))
    out = W_o [ rms_norm(y * silu(z)) in `norm_groups` equal parts, * gain ]

The last taps - 1 projected rows of the convolution's channels live in the slot behind the matrices.

One product makes all columns as float32 sums, the convolution's channels first; `short_conv` reads and writes those
channels alone; `state_space_scan` walks every segment of the step from its slot's matrices (step sizes and decays are
computed there, in float32); `gate_group_norm` gates and norms; the output projection adds into (or fills) the stream.
"""
from __future__ import annotations

import torch

from ..cache import FixedState
from ..config.specs import ConfigError
from ..kernels.api import KernelSet
from .base import Mixer, ParamSpec, register_mixer


@register_mixer("state_space")
class StateSpace(Mixer):
    graph_safe = True
    can_store = True
    kernel_libraries = ("gemm_simt", "scan")

    def __init__(self, ctx, hidden_size: int, num_heads: int, value_dim: int, state_size: int, groups: int, conv_taps: int,
                 norm_groups: int, norm_eps: float):
        """`value_dim`: of a head's x and output; `state_size`: key rows of a head's matrix; `groups`: how many B and C the
        heads share; `conv_taps`: taps of the convolution over time; `norm_groups`: equal parts of the gated output that are
        normed each by its own root mean square, with `norm_eps`."""
        super().__init__(ctx)
        self.d, self.H, self.vd, self.N = int(hidden_size), int(num_heads), int(value_dim), int(state_size)
        self.G, self.taps, self.parts = int(groups), int(conv_taps), int(norm_groups)
        if min(self.d, self.H, self.vd, self.N, self.G, self.parts) < 1 or self.H % self.G:
            raise ConfigError("state_space: sizes must be positive and the heads a multiple of the groups")
        if self.N > 512:
            raise ConfigError(f"state_space: state_size {self.N} exceeds the scan kernel's 512")
        if not 1 <= self.taps <= 8:
            raise ConfigError(f"state_space: conv_taps {conv_taps} must lie in 1..8")
        self.inner = self.H * self.vd
        if self.inner % self.parts:
            raise ConfigError(f"state_space: {self.inner} columns cannot be normed in {self.parts} equal parts")
        if not float(norm_eps) > 0:
            raise ConfigError("state_space: norm_eps must be positive")
        self.eps = float(norm_eps)
        # columns of the product: x, B, C (the convolution's channels), z, a (then padding)
        self.channels = self.inner + 2 * self.G * self.N
        self.b_column, self.c_column = self.inner, self.inner + self.G * self.N
        self.z_column, self.a_column = self.channels, self.channels + self.inner
        self.n_columns = -(-(self.a_column + self.H) // 8) * 8
        self.state_matrices = self.H * KernelSet.scan_state_size(self.N, self.vd)
        self.w_in = self.w_out = self.conv_w = self.conv_b = self.gain = self.a_log = self.dt_bias = self.skip = None

    def param_specs(self):
        return {"in_proj": ParamSpec((2 * self.inner + 2 * self.G * self.N + self.H, self.d)),
                "conv": ParamSpec((self.channels, self.taps)), "conv_bias": ParamSpec((self.channels,)),
                "dt_bias": ParamSpec((self.H,)), "a_log": ParamSpec((self.H,)), "skip": ParamSpec((self.H,), "ones"),
                "norm": ParamSpec((self.inner,), "ones"), "o_proj": ParamSpec((self.d, self.inner))}

    def bind(self, params):
        dt, f32 = self.ctx.dtype, torch.float32
        w = params["in_proj"].to(dt)
        n, c = self.inner, self.channels
        self.w_in = torch.cat([w[n:n + c], w[:n], w[n + c:],
                               torch.zeros((self.n_columns - w.shape[0], self.d), dtype=dt, device=w.device)], 0).contiguous()
        self.w_out = params["o_proj"].to(dt).contiguous()
        self.conv_w, self.conv_b = params["conv"].to(f32).contiguous(), params["conv_bias"].to(f32).contiguous()
        self.gain = params["norm"].to(f32).contiguous()
        self.a_log, self.dt_bias = params["a_log"].to(f32).contiguous(), params["dt_bias"].to(f32).contiguous()
        self.skip = params["skip"].to(f32).contiguous()

    def weight_bytes(self):
        return (self.w_in.numel() + self.w_out.numel()) * self.w_in.element_size() + self.conv_w.numel() * 4

    def cache_request(self):
        # the heads' matrices, then the convolution's rows, rounded up to whole 16-byte groups
        n = self.state_matrices + (self.taps - 1) * self.channels
        return None, FixedState((-(-n // 4) * 4,), torch.float32)

    def forward(self, x, h, batch, cache, accumulate=True):
        k = self.k
        M = x.shape[0]
        proj = torch.empty((M, self.n_columns), dtype=torch.float32, device=x.device)
        k.linear(x, self.w_in, proj)                              # float32 sums: nothing that enters the recurrence is rounded
        u = torch.empty((M, self.channels), dtype=torch.float32, device=x.device)
        k.short_conv(proj, self.conv_w, u, batch, cache.state, channels=self.channels, activation="silu",
                     state_offset=self.state_matrices, bias=self.conv_b)
        y = torch.empty((M, self.inner), dtype=torch.float32, device=x.device)
        k.state_space_scan((u, self.c_column), (u, self.b_column), (u, 0), (proj, self.a_column), y, batch, cache.state,
                           heads=self.H, kv_heads=self.G, dim=self.N, vdim=self.vd, a_log=self.a_log, dt_bias=self.dt_bias,
                           skip=self.skip)
        a = torch.empty((M, self.inner), dtype=x.dtype, device=x.device)
        k.gate_group_norm(y, proj, self.gain, a, groups=self.parts, eps=self.eps, z_column=self.z_column)
        k.linear(a, self.w_out, h, accumulate=accumulate)
