"""Typed configuration of the Zuzadra decoder, read from its config.json.

The file lists the layers one by one: `layers[i]` gives the layer's `type` (which mixer it has), the mixer's sizes and
constants (`mixer`) and its feed-forward (`mlp`, or null for none).  `vocab`, `width`, `norm.eps` and `streams` are the
model's own; `loop` (optional) names a range of layers that run `times` times in a row with the same weights;
`max_positions` and `eos_token_id` are optional.  Every size and every constant that the file gives is read from it;
what the design fixes is stated in `plan()`:

  * `streams` residual streams (hyper-connections): a sublayer reads a weighted sum of them through an RMS norm whose
    weight is stored around zero, and its output, times a learned vector, joins all of them while they mix;
  * mixer `mamba2`: a selective state space with one decay per head, a convolution over time with a bias and silu, the
    output gated and then normed in `norm_groups` equal parts;
  * mixer `parallel`: two mixers on one input, `left_scale` times the left's output plus `right_scale` times the right's.
    Left: grouped-query attention, q and k heads normed with a gain and then rotated in their first `rot.dims` elements
    (element i with i + dims/2), values rotated over the whole value head in the same layout with the same base, heads
    turned back, scores times `scale`, sight of the last `mask.size` positions.  Right: a memory that decays per key
    channel, reading blends of every token with the one before it;
  * feed-forward `dense`: down(xIELU(up x)) with biases and two learned numbers in the activation; an output head of its own.

The inner size of the right mixer's decay (rows of `right.w1`) is not in the file: it is read from the tensor's shape;
where there is no tensor yet (random weights) the optional key `right.rank` gives it, or DEFAULT_RANK.

Tensor names: `embed`, `head`, `final.norm`, and per layer `l<i>.norm1`, `l<i>.norm2`, `l<i>.ls1`, `l<i>.ls2`,
`l<i>.hc<q>.{in,out,mix}`, `l<i>.mix.*` as listed in `weight_bindings`, `l<i>.mlp.{up,up.b,down,down.b,act}`; linear
weights `[out, in]`.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Optional

from .registry import register_architecture
from .specs import BlockSpec, ConfigError, LayerCall, ModelPlan, PartSpec, WeightBinding

DEFAULT_MAX_POSITIONS = 1 << 20
DEFAULT_RANK = 32


def _need(d, key, where):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key `{where}{key}` is missing")
    return d[key]


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                      # taps of the convolution over time
    norm_groups: int


@dataclass(frozen=True)
class WindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]          # mask.size; None: every earlier position is visible
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class DecayMixer:
    heads: int
    dim: int
    rank: Optional[int] = None     # `rank` of the file
    tensor_rank: Optional[int] = None   # what the tensors have

    @property
    def decay_rank(self) -> int:
        return self.tensor_rank or self.rank or DEFAULT_RANK


@dataclass(frozen=True)
class ParallelMixer:
    left: WindowAttention
    right: DecayMixer
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DenseMlp:
    ff: int


@dataclass(frozen=True)
class ZuzadraLayer:
    type: str
    mixer: object                  # StateSpaceMixer | ParallelMixer
    mlp: Optional[DenseMlp]


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@register_architecture("Zuzadra")
@dataclass(frozen=True)
class ZuzadraConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int
    layers: tuple
    loop: Optional[Loop] = None
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Optional[tuple] = None

    MIXERS = ("mamba2", "parallel")

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "ZuzadraConfig":
        layers = []
        for i, L in enumerate(_need(raw, "layers", "")):
            at = f"layers[{i}]."
            kind = _need(L, "type", at)
            m = _need(L, "mixer", at)
            mat = at + "mixer."
            if kind == "mamba2":
                mixer = StateSpaceMixer(**{k: int(_need(m, k, mat)) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")})
            elif kind == "parallel":
                a, b = _need(m, "left", mat), _need(m, "right", mat)
                lat, rat = mat + "left.", mat + "right."
                rot = _need(a, "rot", lat)
                rank = b.get("rank")
                mixer = ParallelMixer(
                    left=WindowAttention(
                        heads=int(_need(a, "heads", lat)), kv_heads=int(_need(a, "kv_heads", lat)), dim=int(_need(a, "dim", lat)),
                        vdim=int(_need(a, "vdim", lat)), scale=float(_need(a, "scale", lat)),
                        window=int(_need(a["mask"], "size", lat + "mask.")) if a.get("mask") else None,
                        rot_dims=int(_need(rot, "dims", lat + "rot.")), rot_base=float(_need(rot, "base", lat + "rot."))),
                    right=DecayMixer(heads=int(_need(b, "heads", rat)), dim=int(_need(b, "dim", rat)),
                                     rank=None if rank is None else int(rank)),
                    left_scale=float(_need(m, "left_scale", mat)), right_scale=float(_need(m, "right_scale", mat)))
            else:
                raise ConfigError(f"config.json: {at}type {kind!r} is not a mixer of this design (known: {', '.join(cls.MIXERS)})")
            f = L.get("mlp")
            mlp = None
            if f is not None:
                fk = _need(f, "kind", at + "mlp.")
                if fk != "dense":
                    raise ConfigError(f"config.json: {at}mlp.kind {fk!r} is unknown (dense)")
                mlp = DenseMlp(ff=int(_need(f, "ff", at + "mlp.")))
            layers.append(ZuzadraLayer(kind, mixer, mlp))
        lp = raw.get("loop")
        loop = None
        if lp is not None:
            loop = Loop(*(int(_need(lp, k, "loop.")) for k in ("start", "stop", "times")))
        eos = raw.get("eos_token_id")
        if isinstance(eos, int):
            eos = (eos,)
        elif eos is not None:
            eos = tuple(int(x) for x in eos)
        cfg = cls(vocab=int(_need(raw, "vocab", "")), width=int(_need(raw, "width", "")),
                  norm_eps=float(_need(_need(raw, "norm", ""), "eps", "norm.")), streams=int(_need(raw, "streams", "")),
                  layers=tuple(layers), loop=loop, max_positions=int(raw.get("max_positions") or DEFAULT_MAX_POSITIONS),
                  eos_token_id=eos)
        cfg.validate()
        return cfg

    def with_tensor_shapes(self, shapes: dict) -> "ZuzadraConfig":
        """The same with the sizes that only the tensors give: the inner size of every right mixer's decay."""
        layers = []
        for i, L in enumerate(self.layers):
            shape = shapes.get(f"l{i}.mix.right.w1")
            if isinstance(L.mixer, ParallelMixer) and shape is not None and len(shape) == 2:
                L = replace(L, mixer=replace(L.mixer, right=replace(L.mixer.right, tensor_rank=int(shape[0]))))
            layers.append(L)
        return replace(self, layers=tuple(layers))

    def validate(self):
        c = self
        for k, v in {"vocab": c.vocab, "width": c.width, "streams": c.streams, "max_positions": c.max_positions}.items():
            if v <= 0:
                raise ConfigError(f"`{k}` must be positive, got {v}")
        if not c.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if not c.layers:
            raise ConfigError("a model needs at least one layer")
        for i, L in enumerate(c.layers):
            m = L.mixer
            at = f"layers[{i}].mixer"
            if isinstance(m, StateSpaceMixer):
                if min(m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) < 1:
                    raise ConfigError(f"{at}: heads, vdim, state, groups, conv and norm_groups must be positive")
                if m.heads % m.groups:
                    raise ConfigError(f"{at}: {m.heads} heads are no multiple of {m.groups} groups")
                if (m.heads * m.vdim) % m.norm_groups:
                    raise ConfigError(f"{at}: {m.heads * m.vdim} columns do not split into norm_groups {m.norm_groups}")
            else:
                a, b = m.left, m.right
                if min(a.heads, a.kv_heads, a.dim, a.vdim, a.window if a.window is not None else 1, b.heads, b.dim) < 1:
                    raise ConfigError(f"{at}: heads, kv_heads, dim, vdim and mask.size must be positive")
                if a.heads % a.kv_heads:
                    raise ConfigError(f"{at}.left: {a.heads} heads are no multiple of {a.kv_heads} kv_heads")
                if not a.scale > 0:
                    raise ConfigError(f"{at}.left: scale must be positive")
                if a.rot_dims < 2 or a.rot_dims % 2 or a.rot_dims > a.dim:
                    raise ConfigError(f"{at}.left: rot.dims {a.rot_dims} must be even and lie in 2..dim ({a.dim})")
                if a.vdim % 2:
                    raise ConfigError(f"{at}.left: vdim {a.vdim} must be even, since the whole value head rotates")
                if not a.rot_base > 0:
                    raise ConfigError(f"{at}.left: rot.base must be positive")
                if b.rank is not None and b.rank < 1:
                    raise ConfigError(f"{at}.right: rank must be positive")
            if L.mlp is not None and L.mlp.ff < 1:
                raise ConfigError(f"layers[{i}].mlp.ff must be positive")
        if c.loop is not None:
            lp = c.loop
            if not 0 <= lp.start < lp.stop <= len(c.layers):
                raise ConfigError(f"loop: layers {lp.start}..{lp.stop - 1} are not a range of the model's {len(c.layers)}")
            if lp.times < 1:
                raise ConfigError("loop.times must be at least 1")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        layers = []
        for L in self.layers:
            m = L.mixer
            if isinstance(m, StateSpaceMixer):
                mixer = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv, "norm_groups": m.norm_groups}
            else:
                a, b = m.left, m.right
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                        "rot": {"base": a.rot_base, "dims": a.rot_dims}}
                if a.window is not None:
                    left["mask"] = {"size": a.window}
                right = {"heads": b.heads, "dim": b.dim}
                if b.rank is not None:
                    right["rank"] = b.rank
                mixer = {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}
            layers.append({"type": L.type, "mixer": mixer, "mlp": None if L.mlp is None else {"kind": "dense", "ff": L.mlp.ff}})
        d = {"architecture": "Zuzadra", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "streams": self.streams, "layers": layers}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    # ------------------------------------------------------------------ the plan
    def run_order(self) -> list:
        """The layers in the order of their runs: those before the loop, the looped range `times` times, the rest."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        lp = self.loop
        return list(range(lp.start)) + list(range(lp.start, lp.stop)) * lp.times + list(range(lp.stop, n))

    def plan(self) -> ModelPlan:
        c = self
        norm = PartSpec("rms_norm", {"size": c.width, "eps": c.norm_eps, "gain_offset": 1.0})
        link = PartSpec("hyper_connection", {"hidden_size": c.width, "streams": c.streams, "layer_scale": True})
        blocks = []
        for L in c.layers:
            m = L.mixer
            if isinstance(m, StateSpaceMixer):
                mixer = PartSpec("state_space", {
                    "hidden_size": c.width, "num_heads": m.heads, "value_dim": m.vdim, "state_size": m.state, "groups": m.groups,
                    "conv_taps": m.conv, "norm_groups": m.norm_groups, "norm_eps": c.norm_eps})
            else:
                a, b = m.left, m.right
                left = PartSpec("paged_attention", {
                    "hidden_size": c.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim,
                    "value_dim": a.vdim, "softmax_scale": a.scale,
                    "window": ("sliding", a.window) if a.window is not None else ("full", 0),
                    "qk_norm_eps": c.norm_eps, "qk_norm_gain": True, "qk_norm_before_rotation": True,
                    "position": PartSpec("rotary_halves", {"rotary_dim": a.rot_dims, "theta": a.rot_base, "exact_angles": True}),
                    "value_rotation": PartSpec("rotary_halves", {"rotary_dim": a.vdim, "theta": a.rot_base, "exact_angles": True})})
                right = PartSpec("decay_memory", {"hidden_size": c.width, "num_heads": b.heads, "head_dim": b.dim,
                                                  "decay_rank": b.decay_rank, "norm_eps": c.norm_eps})
                mixer = PartSpec("parallel_mixers", {"hidden_size": c.width, "left": left, "right": right,
                                                     "left_scale": m.left_scale, "right_scale": m.right_scale})
            parts = {"mixer_norm": norm, "mixer": mixer, "mixer_link": link}
            if L.mlp is not None:
                parts.update(ffn_norm=norm, ffn_link=link, ffn=PartSpec("dense_activation", {
                    "hidden_size": c.width, "intermediate_size": L.mlp.ff, "activation": "xielu", "bias": True}))
            blocks.append(BlockSpec("hyper_residual", parts))
        # every run of a layer has a cache of its own
        order = tuple(LayerCall(i, run, True) for run, i in enumerate(c.run_order()))
        return ModelPlan(hidden_size=c.width, vocab_size=c.vocab, blocks=tuple(blocks), order=order, final_norm=norm,
                         tie_word_embeddings=False, max_positions=c.max_positions, streams=c.streams).validate()

    # ------------------------------------------------------------------ tensor names
    def weight_bindings(self) -> list:
        c = self
        d, n = c.width, c.streams
        B = WeightBinding
        out = [B("embed.weight", "embed", (c.vocab, d)), B("head.weight", "head", (c.vocab, d))]

        def link(place, s, q):
            return [B(f"{place}.in", f"{s}hc{q}.in", (n,), init="ones"), B(f"{place}.out", f"{s}hc{q}.out", (n,), init="ones"),
                    B(f"{place}.mix", f"{s}hc{q}.mix", (n, n)), B(f"{place}.scale", f"{s}ls{q}", (d,), init="ones")]
        for i, L in enumerate(c.layers):
            s, t, m = f"l{i}.", f"layers.{i}.", L.mixer
            x, y = s + "mix.", t + "mixer."
            out.append(B(t + "mixer_norm.weight", s + "norm1", (d,)))
            out += link(t + "mixer_link", s, 1)
            if isinstance(m, StateSpaceMixer):
                inner, ch = m.heads * m.vdim, m.heads * m.vdim + 2 * m.groups * m.state
                out += [B(y + "in_proj", x + "in", (inner + ch + m.heads, d)), B(y + "conv", x + "conv", (ch, m.conv)),
                        B(y + "conv_bias", x + "conv.b", (ch,)), B(y + "dt_bias", x + "dt_bias", (m.heads,)),
                        B(y + "a_log", x + "A_log", (m.heads,)), B(y + "skip", x + "D", (m.heads,), init="ones"),
                        B(y + "norm", x + "norm", (inner,), init="ones"), B(y + "o_proj", x + "o", (d, inner))]
            else:
                a, b = m.left, m.right
                x, y = x + "left.", y + "left."
                out += [B(y + "q_proj", x + "q", (a.heads * a.dim, d)), B(y + "k_proj", x + "k", (a.kv_heads * a.dim, d)),
                        B(y + "v_proj", x + "v", (a.kv_heads * a.vdim, d)), B(y + "q_norm", x + "q.norm", (a.dim,), init="ones"),
                        B(y + "k_norm", x + "k.norm", (a.dim,), init="ones"), B(y + "o_proj", x + "o", (d, a.heads * a.vdim))]
                x, y = s + "mix.right.", t + "mixer.right."
                k = b.heads * b.dim
                out += [B(f"{y}mu_{z}", f"{x}mu.{z}", (d,)) for z in "rkvgw"]
                out += [B(f"{y}{z}_proj", x + z, (k, d)) for z in "rkv"]
                out += [B(y + "gate_proj", x + "g", (k, d)), B(y + "decay_in", x + "w1", (b.decay_rank, d)),
                        B(y + "decay_out", x + "w2", (k, b.decay_rank)), B(y + "decay_bias", x + "w0", (k,)),
                        B(y + "bonus", x + "u", (b.heads, b.dim)), B(y + "norm", x + "norm", (k,), init="ones"),
                        B(y + "o_proj", x + "o", (d, k))]
            if L.mlp is not None:
                f, x, y = L.mlp.ff, s + "mlp.", t + "ffn."
                out.append(B(t + "ffn_norm.weight", s + "norm2", (d,)))
                out += link(t + "ffn_link", s, 2)
                out += [B(y + "up_proj", x + "up", (f, d)), B(y + "up_bias", x + "up.b", (f,)),
                        B(y + "down_proj", x + "down", (d, f)), B(y + "down_bias", x + "down.b", (d,)), B(y + "act", x + "act", (2,))]
        out.append(B("final_norm.weight", "final.norm", (d,)))
        return out

    def unused_tensor_names(self) -> set:
        """What a file may carry for parts this configuration switches off: the second sublayer's of a layer without one."""
        names = set()
        for i, L in enumerate(self.layers):
            if L.mlp is None:
                names |= {f"l{i}.norm2", f"l{i}.ls2", f"l{i}.hc2.in", f"l{i}.hc2.out", f"l{i}.hc2.mix"}
        return names

    checkpoint_prefixes = ("",)
    ignored_prefixes = ()
