"""Typed configuration of the Fozutar decoder, read from its config.json.

The file lists the layers one by one: `layers[i]` gives the layer's `type` (which mixer it has), the mixer's sizes and
constants (`mixer`) and its feed-forward (`mlp`, or null for none).  `vocab`, `width`, `norm.eps`, `embedding.scale` and
`max_positions` are the model's own; `loop` (optional) names a range of layers that run `times` times in a row with the same
weights; `eos_token_id` is optional.  Every size and every constant that the file gives is read from it; what the design
fixes is stated in `plan()`:

  * a layer has one norm, and mixer and feed-forward both read its output and both add to the stream;
  * a learned vector per position is added to the scaled embedding; the output head is the embedding table, unscaled;
  * ahead of pass t through the loop the stream gets the embedding's output (for t > 0) and the pass's vector;
  * mixer `attention`: grouped queries, biases on q and k, the projected keys are the values, q and k heads normed without a
    gain, no rotation, scores times `scale`, squashed to `softcap`, plus a learned number per head and bucket of distances,
    sight limited to the query's chunk of `mask.size` positions;
  * mixer `gla`: gated linear attention, a decay per key channel from two small matrices and the root `tau`;
  * feed-forward `dense`: down(gelu(gate x) * (up x)); `moe`: silu-gated experts, chosen by the largest logits (with a bias)
    and weighted by the softmax over the chosen ones.

Two sizes are not in the file and are read from tensors: the inner size of the decay (rows of `mix.a1`) and the rows of the
table by distance (`mix.rel`).  Where there is no tensor yet (random weights) the optional keys `mixer.rank` and
`mixer.buckets` give them, or DEFAULT_RANK and DEFAULT_BUCKETS.

Tensor names: `embed`, `pos`, `loop.step`, `final.norm`, and per layer `l<i>.norm1`, `l<i>.mix.*` and `l<i>.mlp.*` as listed in
`weight_bindings`; linear weights `[out, in]`.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Optional

from .registry import register_architecture
from .specs import BlockSpec, ConfigError, JunctionCall, LayerCall, ModelPlan, PartSpec, WeightBinding

DEFAULT_RANK = 16
DEFAULT_BUCKETS = 32


def _need(d, key, where):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key `{where}{key}` is missing")
    return d[key]


@dataclass(frozen=True)
class ChunkAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: float
    bias_max: int                  # the distance from which on all keys share the table's last row
    chunk: int                     # mask.size
    buckets: Optional[int] = None  # `buckets` of the file
    tensor_rows: Optional[int] = None   # what the tensor has

    @property
    def table_rows(self) -> int:
        return self.tensor_rows or self.buckets or DEFAULT_BUCKETS


@dataclass(frozen=True)
class GlaMixer:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: Optional[int] = None     # `rank` of the file
    tensor_rank: Optional[int] = None   # what the tensors have

    @property
    def decay_rank(self) -> int:
        return self.tensor_rank or self.rank or DEFAULT_RANK


@dataclass(frozen=True)
class DenseMlp:
    ff: int


@dataclass(frozen=True)
class MoeMlp:
    ff: int                        # of one expert
    experts: int
    top: int


@dataclass(frozen=True)
class FozutarLayer:
    type: str
    mixer: object                  # ChunkAttention | GlaMixer
    mlp: object                    # DenseMlp | MoeMlp | None


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@register_architecture("Fozutar")
@dataclass(frozen=True)
class FozutarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    max_positions: int
    layers: tuple
    loop: Optional[Loop] = None
    eos_token_id: Optional[tuple] = None

    MIXERS = ("attention", "gla")

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "FozutarConfig":
        layers = []
        for i, L in enumerate(_need(raw, "layers", "")):
            at = f"layers[{i}]."
            kind = _need(L, "type", at)
            m = _need(L, "mixer", at)
            mat = at + "mixer."
            optional = lambda key: None if m.get(key) is None else int(m[key])
            if kind == "attention":
                dim, vdim = int(_need(m, "dim", mat)), int(m.get("vdim") or m["dim"])
                if vdim != dim:
                    raise ConfigError(f"config.json: {mat}vdim {vdim} differs from dim {dim}, but the values are the keys")
                mixer = ChunkAttention(
                    heads=int(_need(m, "heads", mat)), kv_heads=int(_need(m, "kv_heads", mat)), dim=dim,
                    scale=float(_need(m, "scale", mat)), softcap=float(_need(m, "softcap", mat)),
                    bias_max=int(_need(m, "bias_max", mat)), chunk=int(_need(_need(m, "mask", mat), "size", mat + "mask.")),
                    buckets=optional("buckets"))
            elif kind == "gla":
                mixer = GlaMixer(heads=int(_need(m, "heads", mat)), dim=int(_need(m, "dim", mat)), vdim=int(_need(m, "vdim", mat)),
                                 tau=float(_need(m, "tau", mat)), rank=optional("rank"))
            else:
                raise ConfigError(f"config.json: {at}type {kind!r} is not a mixer of this design (known: {', '.join(cls.MIXERS)})")
            f = L.get("mlp")
            mlp = None
            if f is not None:
                fat = at + "mlp."
                fk = _need(f, "kind", fat)
                if fk == "dense":
                    mlp = DenseMlp(ff=int(_need(f, "ff", fat)))
                elif fk == "moe":
                    r = _need(f, "router", fat)
                    mlp = MoeMlp(ff=int(_need(_need(f, "expert", fat), "ff", fat + "expert.")),
                                 experts=int(_need(r, "experts", fat + "router.")), top=int(_need(r, "top", fat + "router.")))
                else:
                    raise ConfigError(f"config.json: {fat}kind {fk!r} is unknown (dense, moe)")
            layers.append(FozutarLayer(kind, mixer, mlp))
        lp = raw.get("loop")
        loop = None
        if lp is not None:
            loop = Loop(*(int(_need(lp, k, "loop.")) for k in ("start", "stop", "times")))
        eos = raw.get("eos_token_id")
        if isinstance(eos, int):
            eos = (eos,)
        elif eos is not None:
            eos = tuple(int(x) for x in eos)
        emb = raw.get("embedding") or {}
        cfg = cls(vocab=int(_need(raw, "vocab", "")), width=int(_need(raw, "width", "")),
                  norm_eps=float(_need(_need(raw, "norm", ""), "eps", "norm.")),
                  embedding_scale=float(emb.get("scale", 1.0)), max_positions=int(_need(raw, "max_positions", "")),
                  layers=tuple(layers), loop=loop, eos_token_id=eos)
        cfg.validate()
        return cfg

    def with_tensor_shapes(self, shapes: dict) -> "FozutarConfig":
        """The same with the sizes that only the tensors give: the inner size of every decay, the rows of every table."""
        layers = []
        for i, L in enumerate(self.layers):
            gla = isinstance(L.mixer, GlaMixer)
            shape = shapes.get(f"l{i}.mix.a1" if gla else f"l{i}.mix.rel")
            if shape is not None and len(shape) == 2:
                L = replace(L, mixer=replace(L.mixer, **{"tensor_rank" if gla else "tensor_rows": int(shape[0])}))
            layers.append(L)
        out = replace(self, layers=tuple(layers))
        out.validate()
        return out

    def validate(self):
        c = self
        for k, v in {"vocab": c.vocab, "width": c.width, "max_positions": c.max_positions}.items():
            if v <= 0:
                raise ConfigError(f"`{k}` must be positive, got {v}")
        if not c.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if not c.layers:
            raise ConfigError("a model needs at least one layer")
        for i, L in enumerate(c.layers):
            m, f = L.mixer, L.mlp
            at = f"layers[{i}].mixer"
            if isinstance(m, ChunkAttention):
                if min(m.heads, m.kv_heads, m.dim, m.chunk) < 1 or m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: heads, kv_heads, dim and mask.size must be positive, heads a multiple of kv_heads")
                if not m.scale > 0 or not m.softcap > 0:
                    raise ConfigError(f"{at}: scale and softcap must be positive")
                if m.bias_max < 1 or m.table_rows < 1:
                    raise ConfigError(f"{at}: bias_max and the rows of the table must be positive")
            else:
                if min(m.heads, m.dim, m.vdim, m.decay_rank) < 1:
                    raise ConfigError(f"{at}: heads, dim, vdim and rank must be positive")
                if not m.tau > 0:
                    raise ConfigError(f"{at}: tau must be positive")
            if f is not None and f.ff < 1:
                raise ConfigError(f"layers[{i}].mlp: ff must be positive")
            if isinstance(f, MoeMlp) and (f.experts < 1 or not 1 <= f.top <= f.experts):
                raise ConfigError(f"layers[{i}].mlp.router.top {f.top} must lie in 1..{f.experts}")
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
            m, f = L.mixer, L.mlp
            if isinstance(m, ChunkAttention):
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.dim, "scale": m.scale,
                         "softcap": m.softcap, "bias_max": m.bias_max, "mask": {"size": m.chunk}}
                if m.buckets is not None:
                    mixer["buckets"] = m.buckets
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}
                if m.rank is not None:
                    mixer["rank"] = m.rank
            mlp = None
            if isinstance(f, DenseMlp):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            layers.append({"type": L.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": "Fozutar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale}, "max_positions": self.max_positions, "layers": layers}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.eos_token_id is not None:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    # ------------------------------------------------------------------ the plan
    def run_order(self) -> list:
        """(layer, number of the pass that begins with this run, or None): the layers before the loop, the looped range
        `times` times, the rest."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, None) for i in range(n)]
        out = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            out += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return out + [(i, None) for i in range(lp.stop, n)]

    def plan(self) -> ModelPlan:
        c = self
        norm = PartSpec("rms_norm", {"size": c.width, "eps": c.norm_eps})
        blocks = []
        for L in c.layers:
            m, f = L.mixer, L.mlp
            if isinstance(m, ChunkAttention):
                mixer = PartSpec("paged_attention", {
                    "hidden_size": c.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                    "softmax_scale": m.scale, "score_softcap": m.softcap, "window": ("chunk", m.chunk),
                    "position": PartSpec("no_position"), "qk_norm_eps": c.norm_eps, "bias": True, "output_bias": False,
                    "values_are_keys": True, "distance_table": (m.table_rows, m.bias_max)})
            else:
                mixer = PartSpec("gated_linear_attention", {
                    "hidden_size": c.width, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim,
                    "decay_rank": m.decay_rank, "tau": m.tau, "norm_eps": c.norm_eps})
            parts = {"norm": norm, "mixer": mixer}
            if isinstance(f, DenseMlp):
                parts["ffn"] = PartSpec("dense_swiglu", {"hidden_size": c.width, "intermediate_size": f.ff, "activation": "gelu_tanh"})
            elif f is not None:
                parts["ffn"] = PartSpec("moe_softmax_topk", {"hidden_size": c.width, "num_experts": f.experts, "top_k": f.top,
                                                             "expert_size": f.ff, "router_bias": True})
            blocks.append(BlockSpec("parallel_residual", parts))
        # every run of a layer has a cache or state of its own; a pass through the loop begins with the junction
        order = []
        for run, (i, t) in enumerate(c.run_order()):
            if t is not None:
                order.append(JunctionCall(0, t))
            order.append(LayerCall(i, run, True))
        junctions = () if c.loop is None else (PartSpec("reinject_add", {"hidden_size": c.width, "steps": c.loop.times}),)
        return ModelPlan(hidden_size=c.width, vocab_size=c.vocab, blocks=tuple(blocks), order=tuple(order), final_norm=norm,
                         tie_word_embeddings=True, max_positions=c.max_positions, embedding_scale=c.embedding_scale,
                         position_table=c.max_positions, junctions=junctions).validate()

    # ------------------------------------------------------------------ tensor names
    def weight_bindings(self) -> list:
        c = self
        d = c.width
        B = WeightBinding
        out = [B("embed.weight", "embed", (c.vocab, d)), B("positions.weight", "pos", (c.max_positions, d))]
        if c.loop is not None:
            out.append(B("junctions.0.step", "loop.step", (c.loop.times, d)))
        for i, L in enumerate(c.layers):
            s, t, m, f = f"l{i}.", f"layers.{i}.", L.mixer, L.mlp
            out.append(B(t + "norm.weight", s + "norm1", (d,), init="ones"))
            x, y = s + "mix.", t + "mixer."
            if isinstance(m, ChunkAttention):
                q, k = m.heads * m.dim, m.kv_heads * m.dim
                out += [B(y + "q_proj", x + "q", (q, d)), B(y + "q_bias", x + "q.b", (q,)), B(y + "k_proj", x + "k", (k, d)),
                        B(y + "k_bias", x + "k.b", (k,)), B(y + "distance_bias", x + "rel", (m.table_rows, m.heads)),
                        B(y + "o_proj", x + "o", (d, q))]
            else:
                nk, nv = m.heads * m.dim, m.heads * m.vdim
                out += [B(y + "q_proj", x + "q", (nk, d)), B(y + "k_proj", x + "k", (nk, d)), B(y + "v_proj", x + "v", (nv, d)),
                        B(y + "gate_proj", x + "g", (nv, d)), B(y + "decay_in", x + "a1", (m.decay_rank, d)),
                        B(y + "decay_out", x + "a2", (nk, m.decay_rank)), B(y + "decay_bias", x + "a2.b", (nk,)),
                        B(y + "norm", x + "norm", (m.vdim,), init="ones"), B(y + "o_proj", x + "o", (d, nv))]
            x, y = s + "mlp.", t + "ffn."
            if isinstance(f, DenseMlp):
                out += [B(y + "gate_proj", x + "gate", (f.ff, d)), B(y + "up_proj", x + "up", (f.ff, d)),
                        B(y + "down_proj", x + "down", (d, f.ff))]
            elif f is not None:
                each = lambda name: tuple(f"{x}e{e}.{name}" for e in range(f.experts))
                out += [B(y + "router", x + "router", (f.experts, d)), B(y + "router_bias", x + "router.b", (f.experts,)),
                        B(y + "experts_gate", each("gate"), (f.ff, d)), B(y + "experts_up", each("up"), (f.ff, d)),
                        B(y + "experts_down", each("down"), (d, f.ff))]
        out.append(B("final_norm.weight", "final.norm", (d,), init="ones"))
        return out

    checkpoint_prefixes = ("",)
    ignored_prefixes = ()
