"""Small Fozutar configurations for the tests (none has the sizes of a published model), model folders with random weights,
and the comparison with the plain implementation (`plain_fozutar`)."""
from __future__ import annotations

import functools
from pathlib import Path

import torch

import plain_fozutar as plain
from helpers import note_error
from spite_b200.config import FozutarConfig
from spite_b200.weights import save_file, write_random_model


def _attn(heads, kv, dim, scale, softcap, chunk, far, rows):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap, "bias_max": far,
            "mask": {"size": chunk}, "buckets": rows}


def _gla(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(mixer, mlp=None):
    return {"type": "gla" if "tau" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def _model(vocab, width, eps, emb, positions, layers, loop=None):
    d = {"architecture": "Fozutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb},
         "max_positions": positions, "layers": layers}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# awkward sizes: heads that fill no tensor-core step, a chunk shorter than a page and one across pages, tables that end inside
# the chunk and beyond it, key and value sizes of the memory that are no multiple of four, inner sizes of the decay that are no
# multiple of eight, every kind of feed-forward and none, a loop in the middle that holds both mixers
CONFIG_F = _model(211, 72, 1e-5, 3.0, 400, [
    _layer(_gla(3, 10, 14, 8.0, 5), _dense(40)),
    _layer(_attn(4, 2, 24, 0.3, 4.0, 20, 13, 8), _moe(24, 5, 2)),
    _layer(_gla(2, 33, 7, 16.0, 20)),
    _layer(_attn(3, 3, 10, 0.5, 2.5, 33, 60, 12), _dense(64)),
    _layer(_attn(6, 1, 16, 0.25, 30.0, 50, 31, 6), _moe(40, 3, 3)),
], loop=(1, 4, 3))

# rows of 64 and 128 elements and a width of 128: the tcgen05 and TMA kernels; chunks that cross pages; whole 16-byte groups
# everywhere in the scans, a memory of more than 128 key rows; the loop opens the model
CONFIG_G = _model(520, 128, 1e-6, 7.5, 300, [
    _layer(_attn(4, 2, 64, 0.15, 10.0, 150, 100, 32), _moe(64, 6, 3)),
    _layer(_gla(4, 64, 32, 12.0, 16), _dense(192)),
    _layer(_attn(2, 1, 128, 0.1, 25.0, 64, 40, 16), _dense(128)),
    _layer(_gla(2, 136, 48, 20.0, 72), _moe(128, 4, 1)),
], loop=(0, 2, 2))

# whatever can be one is one: one head, a chunk of one, one expert, one bucket a half, a decay of one number, a loop of one pass
CONFIG_H = _model(97, 40, 1e-3, 1.0, 180, [
    _layer(_gla(1, 8, 6, 1.0, 1), _moe(24, 1, 1)),
    _layer(_attn(1, 1, 8, 1.0, 1.0, 1, 2, 2)),
    _layer(_attn(4, 1, 10, 0.4, 5.0, 7, 3, 4), _dense(8)),
    _layer(_gla(5, 1, 8, 3.0, 3), _moe(8, 4, 4)),
], loop=(0, 4, 1))

# no loop; the table's rows end exactly at whole powers of the ratio between two buckets
CONFIG_J = _model(130, 48, 1e-4, 2.0, 256, [
    _layer(_attn(2, 2, 32, 0.3, 8.0, 90, 64, 8), _dense(56)),
    _layer(_gla(4, 12, 16, 30.0, 8), _moe(32, 8, 2)),
])

CONFIGS = {"F": (CONFIG_F, 0.12, 5), "G": (CONFIG_G, 0.09, 6), "H": (CONFIG_H, 0.2, 7), "J": (CONFIG_J, 0.12, 8)}


def write_model(folder, name: str, dtype=torch.bfloat16, settled_routing=False) -> Path:
    """A model folder with random weights that make every part count: gains away from one, biases and the numbers by distance
    of the size of the scores, decays over their range, position and pass vectors of the embedding's size.
    `settled_routing`: the routers' weights are small and their biases lie half a unit apart in a random order, so that no
    choice of experts is left to rounding (for comparisons in bfloat16); the weights still differ from token to token."""
    cfg, std, seed = CONFIGS[name]
    folder = write_random_model(folder, FozutarConfig.from_dict(cfg), seed=seed, std=std, dtype=dtype)
    _, tensors = plain.load_folder(folder)
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t, s, base=0.0: (base + s * torch.randn(t.shape, generator=g)).to(t.dtype)
    for k, t in tensors.items():
        if k.endswith(("norm", "norm1")):
            tensors[k] = rnd(t, 0.3, 1.0)
        elif k.endswith(".rel"):
            tensors[k] = rnd(t, 1.2)
        elif k.endswith((".q.b", ".k.b")):
            tensors[k] = rnd(t, 0.5)
        elif k.endswith("a2.b"):
            tensors[k] = rnd(t, 2.0, 1.0)
        elif k.endswith(".a2"):
            tensors[k] = (t.float() * 4.0).to(t.dtype)
        elif k.endswith("router.b"):
            tensors[k] = (torch.randperm(t.numel(), generator=g).float() * 0.5).to(t.dtype) if settled_routing else rnd(t, 0.7)
        elif k.endswith("router"):
            tensors[k] = (t.float() * (0.15 if settled_routing else 2.0)).to(t.dtype)
        elif k in ("pos", "loop.step"):
            tensors[k] = rnd(t, 0.6)
    tensors["embed"] = rnd(tensors["embed"], 0.3)
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
    ill-conditioned).  With `sixteen`: the largest distance among two runs whose products' and attention's inputs are
    disturbed by relative errors of up to 2^-7, or four times that of a run that rounds them to bfloat16."""
    key = (str(folder), tuple(tokens), sixteen)
    if key not in _plain_cache:
        cfg, tensors = folder_contents(str(folder))
        run = lambda dtype=torch.float64, r=None: plain.forward(cfg, tensors, list(tokens), dtype, round_inputs=r)
        ref = run()
        g = torch.Generator().manual_seed(len(tokens))
        shaken = lambda size: run(r=lambda x: x * (1.0 + size * (2.0 * torch.rand(x.shape, generator=g, dtype=x.dtype) - 1.0)))
        off = lambda other, times: times * (ref - other.double()).abs().amax(-1)
        if sixteen:
            moved = [off(shaken(2.0 ** -7), 1.0) for _ in range(2)] + [off(run(r=lambda x: x.to(torch.bfloat16).to(x.dtype)), 4.0)]
        else:
            moved = [off(shaken(2.0 ** -23), 8.0) for _ in range(2)] + [off(run(torch.float32), 4.0)]
        _plain_cache[key] = (ref, torch.stack(moved).amax(0) / float(ref.abs().max()))
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
