"""Time mixing with a decay per key channel (the RWKV-6 kind) as a mixer.

Per head a matrix S [dim, dim], zero at the start of a sequence, carried from token to token in float32 in the request's
state slot together with the last token's input:

    m_s = h + (h' - h) mu_s  for s in r, k, v, g, w          h' the token before's h (zeros for the first token)
    r, k, v = W_r m_r, W_k m_k, W_v m_v,   gate = silu(W_g m_g)                              (heads x dim)
    w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))                                                  per head and key channel
    o = (S + diag(u) k v^T)^T r;   S <- diag(w) S + k v^T
    out = W_o [ o_h / rms(o_h) for every head, concatenated, * gain * gate ]

`token_shift` makes the five mixes in one pass; r, k, v and g are one product of four groups with float32 sums; `decay_scan`
computes the decays and the bonus and walks every segment of the step; `head_norm_gate` norms the heads, applies gain and
gate; the output projection adds into (or fills) the stream.
"""
from __future__ import annotations

import torch

from ..cache import FixedState
from ..config.specs import ConfigError
from ..kernels.api import KernelSet
from .base import Mixer, ParamSpec, register_mixer

_MIXES = "rkvgw"


@register_mixer("decay_memory")
class DecayMemory(Mixer):
    graph_safe = True
    can_store = True
    kernel_libraries = ("gemm_simt", "scan")

    def __init__(self, ctx, hidden_size: int, num_heads: int, head_dim: int, decay_rank: int, norm_eps: float):
        """`decay_rank`: rows of the first of the two matrices that make the decay; `norm_eps`: of the heads' norm."""
        super().__init__(ctx)
        self.d, self.H, self.dim, self.rank = int(hidden_size), int(num_heads), int(head_dim), int(decay_rank)
        if min(self.d, self.H, self.dim, self.rank) < 1:
            raise ConfigError("decay_memory: sizes must be positive")
        if self.dim > 512:
            raise ConfigError(f"decay_memory: head_dim {self.dim} exceeds the scan kernel's 512")
        if not float(norm_eps) > 0:
            raise ConfigError("decay_memory: norm_eps must be positive")
        self.eps = float(norm_eps)
        self.n = self.H * self.dim
        self.heads_size = self.n
        self.state_matrices = self.H * KernelSet.scan_state_size(self.dim, self.dim)
        self.w_in = self.w_out = self.w1 = self.w2 = self.mu = self.w0 = self.u = self.gain = None
        self._scaled_gain = {}

    def param_specs(self):
        d, n = self.d, self.n
        specs = {f"mu_{s}": ParamSpec((d,)) for s in _MIXES}
        specs.update({f"{s}_proj": ParamSpec((n, d)) for s in "rkv"})
        specs.update({"gate_proj": ParamSpec((n, d)), "decay_in": ParamSpec((self.rank, d)), "decay_out": ParamSpec((n, self.rank)),
                      "decay_bias": ParamSpec((n,)), "bonus": ParamSpec((self.H, self.dim)), "norm": ParamSpec((n,), "ones"),
                      "o_proj": ParamSpec((d, n))})
        return specs

    def bind(self, params):
        dt, f32 = self.ctx.dtype, torch.float32
        self.w_in = torch.stack([params[s].to(dt) for s in ("r_proj", "k_proj", "v_proj", "gate_proj")], 0).contiguous()
        # (rank and rows of zeros up to a multiple of eight: the tensor-core products take whole 16-byte rows)
        pad = -self.rank % 8
        self.w1 = torch.nn.functional.pad(params["decay_in"].to(dt), (0, 0, 0, pad)).contiguous()
        self.w2 = torch.nn.functional.pad(params["decay_out"].to(dt), (0, pad)).contiguous()
        self.w_out = params["o_proj"].to(dt).contiguous()
        self.mu = torch.stack([params[f"mu_{s}"].to(f32) for s in _MIXES], 0).contiguous()
        self.w0 = params["decay_bias"].to(f32).contiguous()
        self.u = params["bonus"].to(f32).reshape(-1).contiguous()
        self.gain = params["norm"].to(f32).contiguous()
        self._scaled_gain = {1.0: self.gain}

    def gain_times(self, scale: float):
        """The gain with a factor on the whole mixer folded in (float32)."""
        if scale not in self._scaled_gain:
            self._scaled_gain[scale] = (self.gain * scale).contiguous()
        return self._scaled_gain[scale]

    def weight_bytes(self):
        n = self.w_in.numel() + self.w1.numel() + self.w2.numel() + (0 if self.w_out is None else self.w_out.numel())
        return n * self.w_in.element_size()

    def cache_request(self):
        # the heads' matrices, then the last token's input, rounded up to whole 16-byte groups
        n = self.state_matrices + self.d
        return None, FixedState((-(-n // 4) * 4,), torch.float32)

    def heads(self, x, out, column, batch, cache, scale=1.0):
        k = self.k
        M, n, dev = x.shape[0], self.n, x.device
        mixes = torch.empty((len(_MIXES), M, self.d), dtype=x.dtype, device=dev)
        offsets = torch.empty((len(_MIXES) + 1,), dtype=torch.int32, device=dev)
        k.token_shift(x, self.mu, mixes, batch, cache.state, state_offset=self.state_matrices, offsets_out=offsets)
        rkvg = torch.empty((4, M, n), dtype=torch.float32, device=dev)   # float32 sums: nothing that enters the recurrence is rounded
        k.batched_linear(mixes[:4], self.w_in, offsets[:5], rkvg)
        low = torch.empty((M, self.w1.shape[0]), dtype=x.dtype, device=dev)
        k.linear(mixes[4], self.w1, low, activation="tanh")
        w = torch.empty((M, n), dtype=torch.float32, device=dev)
        k.linear(low, self.w2, w)
        o = torch.empty((M, n), dtype=torch.float32, device=dev)
        k.decay_scan((rkvg[0], 0), (rkvg[1], 0), (rkvg[2], 0), w, o, batch, cache.state, heads=self.H, dim=self.dim, vdim=self.dim,
                     w0=self.w0, u=self.u)
        k.head_norm_gate(o, out, heads=self.H, size=self.dim, gates=rkvg[3], gain=self.gain_times(scale), eps=self.eps,
                         gate_activation="silu", out_column=column)

    def forward(self, x, h, batch, cache, accumulate=True):
        a = torch.empty((x.shape[0], self.n), dtype=x.dtype, device=x.device)
        self.heads(x, a, 0, batch, cache)
        self.k.linear(a, self.w_out, h, accumulate=accumulate)
