"""Plain implementation of the Fozutar decoder: whole sequences, no cache, CPU, one function per mechanism, loops where a
loop is the clearest statement.  It shares no code with the package (its own safetensors reader included) and is the
oracle of the Fozutar tests.

The model.  x_0 = E[token] * s_emb + P[position].  Layer: n = N(x), x += mixer(n) + ff(n), one norm in front of both,
N(y) = y / sqrt(mean(y^2) + eps) * gain.  A range of layers may run several times; ahead of pass t the stream gets x_0
(for t > 0) and the vector step[t].  Mixers: `attention` (grouped queries, the projected keys are also the values, biases
on q and k, weightless per-head RMS norm of q and k, scores times a scale, squashed to cap tanh(s / cap), plus a learned
number per head and distance bucket, sight limited to the query's chunk) and `gla` (a matrix per head whose key rows decay
by sigmoid(z)^(1/tau) and take k v^T, read by q after the write; every head normed, gained, gated with silu).
Feed-forward: gelu-gated, or a mixture of silu-gated experts chosen and weighted by the largest router logits.
Output: N(x) E^T.
"""
from __future__ import annotations

import json
import math
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}


def read_safetensors(path) -> dict:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=_DTYPES[info["dtype"]]).reshape(info["shape"]).clone()
    return out


def load_folder(folder):
    with open(f"{folder}/config.json") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(f"{folder}/model.safetensors")


_round = None      # set by `forward(round_inputs=...)`: what an engine that keeps activations in 16 bits does to them


def _in(x):
    """An input of a matrix product (or an attention's q, k, v), rounded the way `forward` was told to."""
    return x if _round is None else _round(x)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bucket(n: int, rows: int, far: int) -> int:
    """The row of a table of `rows` that serves a key n positions back: one row a distance in the first half, then rows
    whose ranges grow geometrically up to the distance `far`, and the last row for everything beyond."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9))


def chunk_visible(T, size):
    """[T, T] bool: query i sees key j <= i of its own chunk, chunks counted from position 0."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def distance_bias(rel, T, far):
    """rel [rows, heads] -> [heads, T, T]: the number added to query i's score of key j <= i (zero elsewhere)."""
    rows = rel.shape[0]
    of = torch.tensor([bucket(n, rows, far) for n in range(T)], dtype=torch.long)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return rel[of[(i - j).clamp(min=0)]].permute(2, 0, 1) * (j <= i)


def attention(h, w, mx, eps):
    T = h.shape[0]
    H, G, dim = mx["heads"], mx["kv_heads"], mx["dim"]
    h = _in(h)
    q = (h @ w["q"].T + w["q.b"]).view(T, H, dim)
    k = (h @ w["k"].T + w["k.b"]).view(T, G, dim)
    v = _in(k)                                               # the projected keys themselves
    q, k = _in(rms(q, eps)), _in(rms(k, eps))
    bias = distance_bias(w["rel"], T, mx["bias_max"])
    sees, cap = chunk_visible(T, mx["mask"]["size"]), mx["softcap"]
    out = torch.zeros(T, H, dim, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * mx["scale"]             # [queries, keys]
        s = cap * torch.tanh(s / cap) + bias[hd]
        out[:, hd] = torch.softmax(s.masked_fill(~sees, -math.inf), -1) @ v[:, g]
    return _in(out.reshape(T, H * dim)) @ w["o"].T


def gla(h, w, mx, eps):
    T = h.shape[0]
    H, dim, vdim = mx["heads"], mx["dim"], mx["vdim"]
    h = _in(h)
    q = (h @ w["q"].T).view(T, H, dim) * dim ** -0.5
    k = (h @ w["k"].T).view(T, H, dim)
    v = (h @ w["v"].T).view(T, H, vdim)
    z = (_in(h @ w["a1"].T) @ w["a2"].T + w["a2.b"]).view(T, H, dim)
    alpha = torch.sigmoid(z) ** (1.0 / mx["tau"])
    gate = silu(h @ w["g"].T)
    S = torch.zeros(H, dim, vdim, dtype=h.dtype)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    out = rms(out, eps) * w["norm"]
    return _in(out.reshape(T, H * vdim) * gate) @ w["o"].T


def dense(h, w, ff):
    h = _in(h)
    return _in(gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def moe(h, w, ff):
    E, top = ff["router"]["experts"], ff["router"]["top"]
    h = _in(h)
    z = h @ w["router"].T + w["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(E), key=lambda e: (-float(z[t, e]), e))[:top]
        share = torch.softmax(z[t, order], 0)
        for s, e in zip(share, order):
            a = _in(silu(h[t] @ w[f"e{e}.gate"].T) * (h[t] @ w[f"e{e}.up"].T))
            out[t] += s * (a @ w[f"e{e}.down"].T)
    return out


MIXERS = {"attention": attention, "gla": gla}
FEED_FORWARDS = {"dense": dense, "moe": moe}


def _sub(tensors, prefix, dtype):
    return {k[len(prefix):]: v.to(dtype) for k, v in tensors.items() if k.startswith(prefix)}


def runs(cfg):
    """[(layer, pass or None)]: every run of a layer; a number marks the first layer of that pass through the loop."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if lp is None:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        out += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return out + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, tensors, tokens, dtype=torch.float32, taps=None, round_inputs=None):
    """Logits [T, vocab] of one sequence; `taps`, a list, receives the residual stream after every layer run;
    `round_inputs`, a function, is applied to every input of a matrix product and to attention's q, k and v."""
    global _round
    _round = round_inputs
    try:
        return _forward(cfg, tensors, tokens, dtype, taps)
    finally:
        _round = None


def _forward(cfg, tensors, tokens, dtype, taps):
    eps = cfg["norm"]["eps"]
    E = tensors["embed"].to(dtype)
    T = len(tokens)
    x = E[torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"] + tensors["pos"][:T].to(dtype)
    x0 = x.clone()
    for i, t in runs(cfg):
        if t is not None:
            if t > 0:
                x = x + x0
            x = x + tensors["loop.step"][t].to(dtype)
        L, p = cfg["layers"][i], f"l{i}."
        n = rms_norm(x, tensors[p + "norm1"].to(dtype), eps)
        y = MIXERS[L["type"]](n, _sub(tensors, p + "mix.", dtype), L["mixer"], eps)
        if L.get("mlp") is not None:
            y = y + FEED_FORWARDS[L["mlp"]["kind"]](n, _sub(tensors, p + "mlp.", dtype), L["mlp"])
        x = x + y
        if taps is not None:
            taps.append(x.clone())
    return _in(rms_norm(x, tensors["final.norm"].to(dtype), eps)) @ E.T
