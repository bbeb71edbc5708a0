"""Small Zuzadra configurations for the tests (none has the sizes of a published model), model folders with random
weights, and the comparison with the plain implementation (`plain_zuzadra`)."""
from __future__ import annotations

import functools
from pathlib import Path

import torch

import plain_zuzadra as plain
from helpers import note_error
from spite_b200.config import ZuzadraConfig
from spite_b200.weights import save_file, write_random_model


def _ssm(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _left(heads, kv, dim, vdim, scale, dims, base, window=None):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if window is not None:
        d["mask"] = {"size": window}
    return d


def _par(left, heads, dim, rank, left_scale, right_scale):
    return {"left": left, "right": {"heads": heads, "dim": dim, "rank": rank}, "left_scale": left_scale, "right_scale": right_scale}


def _layer(mixer, ff=None):
    return {"type": "parallel" if "left" in mixer else "mamba2", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _model(vocab, width, eps, streams, layers, loop=None):
    d = {"architecture": "Zuzadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# awkward sizes: value heads smaller and larger than key heads, rotations of 6 and of the whole head, windows shorter than a
# page and across pages and none, several groups of B and C, several norm parts, state sizes that are no multiple of four, a
# rank that is no multiple of eight, a looped range in the middle, layers without a feed-forward, two streams
CONFIG_P = _model(211, 72, 1e-5, 2, [
    _layer(_ssm(6, 20, 18, groups=3, conv=3, norm_groups=4), ff=96),
    _layer(_par(_left(4, 2, 24, 16, 0.2, 6, 50.0, window=20), 3, 10, 5, 0.7, 1.2), ff=40),
    _layer(_ssm(2, 7, 40, groups=2, conv=1, norm_groups=2)),
    _layer(_par(_left(3, 3, 16, 30, 0.25, 16, 10000.0), 2, 33, 12, 1.3, 0.4)),
    _layer(_ssm(1, 36, 5, conv=8), ff=64),
], loop=(1, 4, 3))

# rows of 64 and 128 elements and a width of 128: the tcgen05 and TMA kernels; windows of a page and of more; value heads of 96
# in rows of 128; whole 16-byte groups everywhere in the scans, heads of more than 128 key rows; four streams
CONFIG_Q = _model(520, 128, 1e-6, 4, [
    _layer(_par(_left(4, 2, 64, 64, 0.125, 32, 1e6, window=150), 4, 64, 16, 0.9, 0.8), ff=192),
    _layer(_ssm(8, 32, 64, groups=2, conv=4, norm_groups=2), ff=128),
    _layer(_par(_left(2, 1, 128, 96, 0.09, 64, 500.0, window=64), 2, 136, 24, 1.0, 1.0), ff=256),
    _layer(_ssm(2, 64, 128, conv=2), ff=128),
], loop=(0, 2, 2))

# whatever can be one is one: one head, one group, a window of one, one tap, one stream, a loop of one pass
CONFIG_R = _model(97, 40, 1e-3, 1, [
    _layer(_par(_left(1, 1, 8, 6, 0.4, 2, 10.0, window=1), 1, 8, 1, 1.0, -0.5), ff=24),
    _layer(_ssm(1, 1, 1, conv=1), ff=1),
    _layer(_par(_left(4, 1, 10, 8, 0.3, 4, 100.0, window=7), 5, 1, 3, -1.1, 1.0)),
], loop=(0, 3, 1))

# five streams, no loop, the state space alone but for one layer
CONFIG_S = _model(130, 48, 1e-4, 5, [
    _layer(_ssm(4, 12, 16, groups=4, conv=4, norm_groups=3), ff=32),
    _layer(_par(_left(2, 2, 32, 32, 0.2, 32, 1000.0, window=33), 3, 16, 8, 0.6, 0.9), ff=56),
])

CONFIGS = {"P": (CONFIG_P, 0.12, 5), "Q": (CONFIG_Q, 0.09, 6), "R": (CONFIG_R, 0.2, 7), "S": (CONFIG_S, 0.12, 8)}


def write_model(folder, name: str, dtype=torch.bfloat16) -> Path:
    """A model folder with random weights that make every part count: gains and coefficients of the streams away from their
    neutral values, streams that stay bounded while they mix, state-space decays and channel decays over their range."""
    cfg, std, seed = CONFIGS[name]
    folder = write_random_model(folder, ZuzadraConfig.from_dict(cfg), seed=seed, std=std, dtype=dtype)
    _, tensors = plain.load_folder(folder)
    g = torch.Generator().manual_seed(seed)
    n = int(cfg["streams"])
    rnd = lambda t, s, base=0.0: (base + s * torch.randn(t.shape, generator=g)).to(t.dtype)
    for k, t in tensors.items():
        last = k.split(".", 1)[-1]
        if last.endswith("norm") or ".ls" in k:
            tensors[k] = rnd(t, 0.3, 1.0)
        elif ".norm1" in k or ".norm2" in k or k == "final.norm":
            tensors[k] = rnd(t, 0.3)
        elif last in ("hc1.in", "hc2.in"):
            tensors[k] = rnd(t, 0.4, 1.0 / n)
        elif last in ("hc1.out", "hc2.out"):
            tensors[k] = rnd(t, 0.4, 0.8)
        elif last in ("hc1.mix", "hc2.mix"):
            tensors[k] = (0.75 * torch.eye(n) + (0.25 / n) * (1.0 + torch.randn((n, n), generator=g))).to(t.dtype)
        elif last.endswith(("A_log", "w0")):
            tensors[k] = rnd(t, 1.0, -1.0)
        elif last.endswith(("dt_bias", "right.u", ".D", "conv.b", "up.b", "down.b", "mlp.act")):
            tensors[k] = rnd(t, 0.5)
        elif last.endswith("mix.conv"):
            tensors[k] = rnd(t, 0.5)
        elif ".mu." in k:
            tensors[k] = torch.rand(t.shape, generator=g).to(t.dtype)
        elif last.endswith("right.w2"):
            tensors[k] = (t.float() * 4.0).to(t.dtype)
    tensors["embed"] = rnd(tensors["embed"], 1.0)
    save_file(tensors, Path(folder) / "model.safetensors")
    return Path(folder)


@functools.lru_cache(maxsize=None)
def folder_contents(folder: str):
    return plain.load_folder(folder)


_plain_cache: dict = {}


def plain_logits(folder, tokens, sixteen=False):
    """(logits computed in float64, what a position may be off by through rounding alone, as a fraction of the largest
    logit).  For float32 arithmetic: four times the distance of a float32 run, or eight times that of a run whose products'
    inputs are disturbed by relative errors of up to 2^-23 (a head of a memory that puts out next to nothing before its norm is
    ill-conditioned).  With `sixteen`: the largest distance among
    two runs whose products' and attention's inputs are disturbed by relative errors of up to 2^-7, or four times that of a
    run that rounds them to bfloat16."""
    key = (str(folder), tuple(tokens), sixteen)
    if key not in _plain_cache:
        cfg, tensors = folder_contents(str(folder))
        ref = plain.forward(cfg, tensors, list(tokens), torch.float64)
        if sixteen:
            g = torch.Generator().manual_seed(len(tokens))
            shake = lambda x: x * (1.0 + 2.0 ** -7 * (2.0 * torch.rand(x.shape, generator=g, dtype=x.dtype) - 1.0))
            lows = [plain.forward(cfg, tensors, list(tokens), torch.float64, round_inputs=shake) for _ in range(2)]
            exact = plain.forward(cfg, tensors, list(tokens), torch.float64, round_inputs=lambda x: x.to(torch.bfloat16).to(x.dtype))
            moved = torch.stack([(ref - low).abs().amax(-1) for low in lows] + [4.0 * (ref - exact).abs().amax(-1)]).amax(0)
        else:
            g = torch.Generator().manual_seed(len(tokens))
            shake = lambda x: x * (1.0 + 2.0 ** -23 * (2.0 * torch.rand(x.shape, generator=g, dtype=x.dtype) - 1.0))
            lows = [plain.forward(cfg, tensors, list(tokens), torch.float64, round_inputs=shake) for _ in range(3)]
            moved = torch.stack([8.0 * (ref - low).abs().amax(-1) for low in lows] +
                                [4.0 * (ref - plain.forward(cfg, tensors, list(tokens), torch.float32).double()).abs().amax(-1)]).amax(0)
        _plain_cache[key] = (ref, moved / float(ref.abs().max()))
    return _plain_cache[key]


def generate_greedy(cfg, tensors, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(plain.forward(cfg, tensors, toks)[-1])))
    return toks[len(prompt):]


def compare_with_plain(results: dict, folder, requests: dict, tol: float):
    """Every logits row against the plain implementation in float64, as a fraction of the largest logit of the sequence;
    names the first position beyond its allowance: `tol`, or what `plain_logits` finds that rounding alone may do there.
    In the 16-bit comparison (a `tol` of a thousandth or more) one position in twenty-five of a request (or two) may be off
    by up to three times its allowance: the estimate is a few draws."""
    worst = 0.0
    sixteen = tol >= 1e-3
    for r, toks in requests.items():
        ref, rounding = plain_logits(folder, toks, sixteen=sixteen)
        scale = float(ref.abs().max())
        spare = max(2, len(toks) // 25) if sixteen else 0
        for p in range(len(toks)):
            if (r, p) not in results:
                continue
            err = float((results[(r, p)].double().cpu() - ref[p]).abs().max()) / scale
            allowed = max(tol, float(rounding[p]))
            if allowed < err <= 3.0 * allowed and spare > 0:
                spare -= 1
                continue
            worst = max(worst, err * tol / allowed)
            assert err <= allowed, (f"request {r!r}, position {p} (first wrong one): error {err:.3e} of the "
                                    f"logit scale exceeds {allowed:.1e} (worst before it: {worst:.3e})")
    note_error(worst, tol)
    return worst
