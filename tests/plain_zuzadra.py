"""Plain, slow implementation of the Zuzadra decoder: whole sequences, no cache, float32 (or float64) on the CPU, one
function per mechanism, written from the design's equations.  It shares no code with the package: it has its own
safetensors reader and takes the parsed config.json as a dict.

Notation: X is the list of residual streams, each [T, d], of one sequence; h a sublayer's input, p a position (from 0).
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch


# ---------------------------------------------------------------------------------- files
def read_safetensors(path) -> dict:
    """8-byte little-endian header length, JSON header (name -> dtype, shape, data_offsets), data."""
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = memoryview(raw)[8 + n:]
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
    return out


def load_folder(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# ---------------------------------------------------------------------------------- mechanisms
_round = None        # `forward(round_inputs=...)`: applied to the activations that enter every matrix product and to what attention reads and writes


def _in(x):
    return x if _round is None else _round(x)


def unit_rms(x, eps):
    """x over its root mean square: x / sqrt(mean(x^2) + eps), along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """A norm whose weight is stored around zero: the gain is 1 + w."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def xielu(z, p, q):
    """z > 0: softplus(p) z^2 + z / 2; else (1/2 + softplus(q)) (e^z - 1 - z) + z / 2."""
    neg = torch.clamp(z, max=0)
    return torch.where(z > 0, softplus(p) * z * z + 0.5 * z, (0.5 + softplus(q)) * (torch.expm1(neg) - neg) + 0.5 * z)


def dense_ff(h, w):
    a = xielu(_in(h) @ w["up"].T + w["up.b"], w["act"][0], w["act"][1])
    return _in(a) @ w["down"].T + w["down.b"]


def rotate_halves(x, dims, base, sign=1.0):
    """x [T, heads, size]: element i < dims/2 of every head pairs with i + dims/2; the pair (u, v) of position p turns by
    a = sign p base^(-2i/dims): (u cos a - v sin a, v cos a + u sin a).  Elements from `dims` on pass."""
    T = x.shape[0]
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = sign * torch.arange(T, dtype=torch.float64)[:, None] * f[None, :]
    cos, sin = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def window_mask(T, size):
    """[T, T] True where row i may see column j: 0 <= i - j < size (no size: j <= i)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def attention(h, w, mx, eps):
    """Grouped-query attention: heads normed with a gain of their own size, leading elements rotated, values rotated by
    their own position over the whole value head, the heads' results turned back by the query's position."""
    T = h.shape[0]
    h = _in(h)
    H, G, dim, vdim = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    dims, base = int(mx["rot"]["dims"]), float(mx["rot"]["base"])
    q = _in((h @ w["q"].T).reshape(T, H, dim))
    k = _in((h @ w["k"].T).reshape(T, G, dim))
    v = _in((h @ w["v"].T).reshape(T, G, vdim))
    q = _in(rotate_halves(unit_rms(q, eps) * w["q.norm"], dims, base))
    k = _in(rotate_halves(unit_rms(k, eps) * w["k.norm"], dims, base))
    v = _in(rotate_halves(v, vdim, base))
    see = window_mask(T, int(mx["mask"]["size"]) if mx.get("mask") else None)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * float(mx["scale"])
        out[:, a] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    out = rotate_halves(_in(out), vdim, base, sign=-1.0)
    return _in(out.reshape(T, H * vdim)) @ w["o"].T


def decay_attention(h, w, mx, eps):
    """Time mixing with a decay per key channel.  Every one of r, k, v, g, w reads h + (h' - h) mu, h' the token before's h.
    Per head: o_t = (S_(t-1) + diag(u) k v^T)^T r, then S_t = diag(w) S_(t-1) + k v^T."""
    T, d = h.shape
    h = _in(h)
    H, dim = int(mx["heads"]), int(mx["dim"])
    before = torch.cat([torch.zeros(1, d, dtype=h.dtype), h[:-1]], 0)
    mix = {s: _in(h + (before - h) * w["mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).reshape(T, H, dim) for s in "rkv")
    gate = silu(mix["g"] @ w["g"].T)
    z = _in(torch.tanh(mix["w"] @ w["w1"].T)) @ w["w2"].T + w["w0"]
    decay = torch.exp(-torch.exp(z)).reshape(T, H, dim)
    out = torch.zeros(T, H, dim, dtype=h.dtype)
    S = torch.zeros(H, dim, dim, dtype=h.dtype)
    u = w["u"]
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    out = unit_rms(out, eps).reshape(T, H * dim) * w["norm"] * gate
    return _in(out) @ w["o"].T


def parallel(h, w, mx, eps):
    left = attention(h, _sub(w, "left."), mx["left"], eps)
    right = decay_attention(h, _sub(w, "right."), mx["right"], eps)
    return float(mx["left_scale"]) * left + float(mx["right_scale"]) * right


def causal_conv(x, w, bias):
    """x [T, C], w [C, taps] (the last column is the current token's), zeros before the start."""
    T, C = x.shape
    n = w.shape[1]
    padded = torch.cat([torch.zeros(n - 1, C, dtype=x.dtype), x], 0)
    return sum(padded[j:j + T] * w[:, j] for j in range(n)) + bias


def state_space(h, w, mx, eps):
    """S_t = exp(-exp(A_log) dt) S_(t-1) + dt B x^T (per head; B and C shared by a group of heads), y = S_t^T C + D x;
    then times silu(z), normed in equal parts, times the gain."""
    T = h.shape[0]
    h = _in(h)
    H, P, N, G = int(mx["heads"]), int(mx["vdim"]), int(mx["state"]), int(mx["groups"])
    inner = H * P
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w["dt_bias"])                                     # [T, H]
    keep = torch.exp(-torch.exp(w["A_log"]) * dt)
    out = torch.zeros(T, H, P, dtype=h.dtype)
    S = torch.zeros(H, N, P, dtype=h.dtype)
    of = torch.arange(H) // (H // G)
    for t in range(T):
        S = keep[t][:, None, None] * S + dt[t][:, None, None] * B[t, of][:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, C[t, of]) + w["D"][:, None] * x[t]
    y = out.reshape(T, inner) * silu(z)
    parts = int(mx["norm_groups"])
    y = unit_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w["norm"]
    return _in(y) @ w["o"].T


MIXERS = {"mamba2": state_space, "parallel": parallel}


# ---------------------------------------------------------------------------------- the streams
def gather_streams(X, w_in):
    """u = sum_s w_in[s] x_s"""
    return sum(w_in[s] * X[s] for s in range(len(X)))


def mix_streams(X, y, mix, w_out):
    """x_t <- sum_s mix[s, t] x_s + w_out[t] y, all from the old ones."""
    n = len(X)
    return [sum(mix[s, t] * X[s] for s in range(n)) + w_out[t] * y for t in range(n)]


# ---------------------------------------------------------------------------------- the model
def _sub(tensors, prefix, dtype=None):
    return {k[len(prefix):]: v if dtype is None else v.to(dtype) for k, v in tensors.items() if k.startswith(prefix)}


def run_order(cfg):
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b, times = int(lp["start"]), int(lp["stop"]), int(lp["times"])
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def forward(cfg, tensors, tokens, dtype=torch.float32, taps=None, round_inputs=None):
    """Logits [T, vocab] of one whole sequence.  `taps`, a list, receives the sum of the streams after every layer run.
    `round_inputs`, a function, is applied to the activations that enter every matrix product, to queries, keys and
    values as attention reads them and to the heads it puts out (and to nothing else): with a rounding to 16 bits it
    shows how far that rounding alone moves the logits."""
    global _round
    _round = round_inputs
    try:
        return _forward(cfg, tensors, tokens, dtype, taps)
    finally:
        _round = None


def _forward(cfg, tensors, tokens, dtype, taps):
    eps = float(cfg["norm"]["eps"])
    x0 = tensors["embed"].to(dtype)[torch.tensor(tokens, dtype=torch.long)]
    X = [x0.clone() for _ in range(int(cfg["streams"]))]
    for i in run_order(cfg):
        layer = cfg["layers"][i]
        w = _sub(tensors, f"l{i}.", dtype)
        u = gather_streams(X, w["hc1.in"])
        y = MIXERS[layer["type"]](offset_norm(u, w["norm1"], eps), _sub(w, "mix."), layer["mixer"], eps)
        X = mix_streams(X, w["ls1"] * y, w["hc1.mix"], w["hc1.out"])
        if layer.get("mlp") is not None:
            u = gather_streams(X, w["hc2.in"])
            y = dense_ff(offset_norm(u, w["norm2"], eps), _sub(w, "mlp."))
            X = mix_streams(X, w["ls2"] * y, w["hc2.mix"], w["hc2.out"])
        if taps is not None:
            taps.append(sum(X))
    x = _in(offset_norm(sum(X), tensors["final.norm"].to(dtype), eps))
    return x @ tensors["head"].to(dtype).T
