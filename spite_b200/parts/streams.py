"""Several residual streams instead of one (hyper-connections).

A model of n streams x_1 .. x_n (all equal to the embedding's output at the start) runs a sublayer on a weighted sum of
them and lays its output back into all of them, while they mix:

    u = sum_s in[s] x_s;   y = sublayer(norm(u)) * scale;   x_t <- sum_s mix[s, t] x_s + out[t] y   (all from the old ones)

At the end the stream is their sum.  `ResidualStreams` is what the layers of such a model hand on in place of the one
stream h; `HyperConnection` holds a sublayer's coefficients; the arrangement `hyper_residual` is a layer of two such
sublayers.  A sublayer's output is not laid into the streams at once: it waits until the streams are read next, and one
kernel (`KernelSet.streams`) then mixes, adds, forms the next u and norms it.
"""
from __future__ import annotations

import torch

from ..config.specs import ConfigError
from .base import Block, ParamSpec, Part, register_block, register_connection


class ResidualStreams:
    """x float32 [tokens, n, d] and, possibly, a sublayer's output that is still to be laid into them."""

    def __init__(self, kernels, x):
        self.k, self.x = kernels, x
        self.pending = None

    @property
    def shape(self):
        return (self.x.shape[0], self.x.shape[2])

    @property
    def device(self):
        return self.x.device

    def leave(self, y, link, bias=None):
        """The sublayer behind the connection `link` has put out y [tokens, d]."""
        self.settle()
        self.pending = dict(y=y, bias=bias, scale=link.scale, mix=link.mix, w_out=link.w_out)

    def enter(self, w_in, norm, out, rows=None, last=False):
        """out = norm(sum_s w_in[s] x_s); `last`: nobody reads the streams afterwards (they need not be stored)."""
        pending, self.pending = self.pending, None
        self.k.streams(self.x, **(pending or {}), w_in=w_in, gain=None if norm is None else norm.weight,
                       eps=None if norm is None else norm.eps, next_out=out, rows=rows, write_back=not last)

    def settle(self):
        if self.pending is not None:
            pending, self.pending = self.pending, None
            self.k.streams(self.x, **pending)

    def total(self):
        """The sum of the streams, float32 [tokens, d]."""
        self.settle()
        out = torch.empty(self.shape, dtype=torch.float32, device=self.device)
        self.k.streams(self.x, w_in=torch.ones(self.x.shape[1], dtype=torch.float32, device=self.device), next_out=out)
        return out


@register_connection("hyper_connection")
class HyperConnection(Part):
    """The coefficients of one sublayer: `in` [n], `out` [n], `mix` [n, n] ([from, to]) and, with `layer_scale`, `scale` [d]
    on the sublayer's output."""
    graph_safe = True
    kernel_libraries = ("elementwise",)

    def __init__(self, ctx, hidden_size: int, streams: int, layer_scale: bool = False):
        super().__init__(ctx)
        self.d, self.n, self.layer_scale = int(hidden_size), int(streams), bool(layer_scale)
        if not 1 <= self.n <= 32:
            raise ConfigError(f"hyper_connection: {streams} streams must lie in 1..32")
        self.w_in = self.w_out = self.mix = self.scale = None

    def param_specs(self):
        specs = {"in": ParamSpec((self.n,), "ones"), "out": ParamSpec((self.n,), "ones"), "mix": ParamSpec((self.n, self.n))}
        if self.layer_scale:
            specs["scale"] = ParamSpec((self.d,), "ones")
        return specs

    def bind(self, params):
        f32 = torch.float32
        self.w_in, self.w_out = params["in"].to(f32).contiguous(), params["out"].to(f32).contiguous()
        self.mix = params["mix"].to(f32).contiguous()
        self.scale = params["scale"].to(f32).contiguous() if self.layer_scale else None

    def weight_bytes(self):
        return (self.n * (self.n + 2) + (self.d if self.layer_scale else 0)) * 4


@register_block("hyper_residual")
class HyperResidual(Block):
    """A layer of one or two sublayers on several residual streams."""
    graph_safe = True
    places = {"mixer_norm": "norm", "mixer": "mixer", "mixer_link": "connection",
              "ffn_norm": "norm", "ffn": "feed_forward", "ffn_link": "connection"}
    optional = ("ffn_norm", "ffn", "ffn_link")

    def __init__(self, ctx, spec):
        super().__init__(ctx, spec)
        if self.ffn is not None and (self.ffn_norm is None or self.ffn_link is None):
            raise ConfigError("hyper_residual: a feed-forward needs its norm and its connection")
        for n in (self.mixer_norm, self.ffn_norm):
            if n is not None and n.kind != "rms_norm":
                raise ConfigError("hyper_residual fuses its norms with the streams' mixing: RMS norms")

    def _output(self, part, x, *args):
        y = torch.empty(x.shape, dtype=torch.float32, device=x.device)
        bias = getattr(part, "output_bias", None)
        if part.can_store:
            part.forward(x, y, *args, accumulate=False, **({"add_bias": False} if bias is not None else {}))
        else:
            y.zero_()
            part.forward(x, y, *args)
            bias = None                       # (added by the part itself)
        return y, bias

    def forward(self, h, batch, cache):
        x = torch.empty(h.shape, dtype=self.ctx.dtype, device=h.device)
        h.enter(self.mixer_link.w_in, self.mixer_norm, x)
        y, bias = self._output(self.mixer, x, batch, cache)
        h.leave(y, self.mixer_link, bias)
        if self.ffn is not None:
            x = torch.empty(h.shape, dtype=self.ctx.dtype, device=h.device)
            h.enter(self.ffn_link.w_in, self.ffn_norm, x)
            y, bias = self._output(self.ffn, x, batch)
            h.leave(y, self.ffn_link, bias)
