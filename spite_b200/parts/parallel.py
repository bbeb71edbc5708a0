"""Two mixers side by side on the same input: left_scale * left(x) + right_scale * right(x).

Both mixers end in an output projection, so the sum is one product over the concatenated heads: the mixers write their
heads, each times its scale (applied in float32 before the heads are rounded), into the columns of one buffer, and one
matrix [W_left | W_right] adds both into (or fills) the stream.  The layer's cache is what the two ask for together: at
most one may keep pages and at most one a state slot.  On a GPU the right mixer runs on a side stream beside the left.
"""
from __future__ import annotations

import torch

from ..config.specs import ConfigError, PartSpec
from .base import Mixer, ParamSpec, build_part, register_mixer, side_stream


@register_mixer("parallel_mixers")
class ParallelMixers(Mixer):
    can_store = True

    def __init__(self, ctx, hidden_size: int, left: PartSpec, right: PartSpec, left_scale: float = 1.0, right_scale: float = 1.0):
        super().__init__(ctx)
        self.d = int(hidden_size)
        self.sides = {"left": build_part("mixer", left, ctx), "right": build_part("mixer", right, ctx)}
        self.scales = {"left": float(left_scale), "right": float(right_scale)}
        for name, m in self.sides.items():
            if m.heads_size is None:
                raise ConfigError(f"parallel_mixers: the {name} mixer {m.kind!r} does not end in one plain output projection")
        self.n_left, self.n = self.sides["left"].heads_size, sum(m.heads_size for m in self.sides.values())
        self.kernel_libraries = tuple(sorted({lib for m in self.sides.values() for lib in m.kernel_libraries}))
        self.graph_safe = all(m.graph_safe for m in self.sides.values())
        self.side_by_side = True              # the right mixer on a side stream
        self.wo = None
        self.cache_request()                  # (two mixers that want the same kind of cache are refused here)

    def param_specs(self):
        return {f"{side}.{n}": s for side, m in self.sides.items() for n, s in m.param_specs().items()}

    def bind(self, params):
        outs = []
        for side, m in self.sides.items():
            own = {n[len(side) + 1:]: t for n, t in params.items() if n.startswith(side + ".")}
            m.bind(own)
            m.drop_output_projection()
            outs.append(own["o_proj"].to(self.ctx.dtype))
        self.wo = torch.cat(outs, 1).contiguous()

    def weight_bytes(self):
        return self.wo.numel() * self.wo.element_size() + sum(m.weight_bytes() for m in self.sides.values())

    def cache_request(self):
        wants = [m.cache_request() for m in self.sides.values()]
        kv = [a for a, _ in wants if a is not None]
        state = [b for _, b in wants if b is not None]
        if len(kv) > 1 or len(state) > 1:
            raise ConfigError("parallel_mixers: both mixers ask for the same kind of cache")
        return (kv or [None])[0], (state or [None])[0]

    def forward(self, x, h, batch, cache, accumulate=True):
        a = torch.empty((x.shape[0], self.n), dtype=x.dtype, device=x.device)
        left, right = self.sides["left"], self.sides["right"]
        side = side_stream(x) if self.side_by_side else None
        if side is not None:
            main = torch.cuda.current_stream(x.device)
            forked = torch.cuda.Event()
            forked.record(main)
            with torch.cuda.stream(side):
                side.wait_event(forked)
                right.heads(x, a, self.n_left, batch, cache, self.scales["right"])
                done = torch.cuda.Event()
                done.record(side)
            left.heads(x, a, 0, batch, cache, self.scales["left"])
            main.wait_event(done)
        else:
            left.heads(x, a, 0, batch, cache, self.scales["left"])
            right.heads(x, a, self.n_left, batch, cache, self.scales["right"])
        self.k.linear(a, self.wo, h, accumulate=accumulate)
