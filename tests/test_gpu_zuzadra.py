"""Zuzadra on the GPU.  First every new mechanism alone against loops written here from its equation, in float64 (the two scans
in prompts, portions and decoded tokens with a far token and slots used again, the token shift, the convolution's bias, the
gate before a norm in parts, several residual streams, rotated values and heads turned back, far angles, biases and xIELU in
every product kernel, one product per group, windows with keys just inside and outside); then the engine in float32 and
bfloat16 against the plain implementation in every cut (whole, token by token, portions down to two tokens, mixed batches in a
pool whose pages and slots are used again, free pages poisoned), layer run by layer run, long decoding, captured steps with
padding rows, greedy generation through `LLM.generate`, `bin/trace_run` and the command line."""
import json
import math

import pytest
import torch

import helpers as H
import plain_zuzadra as plain
import zuzadra_helpers as S
from reference_kernels import TorchReferenceKernels
from spite_b200.cache import LayerCache, Window
from spite_b200.engine.batch import Segment, build_step_batch
from spite_b200.parts import QkNorm, Rotation
from test_gpu_kernels import close, fill_cache, make_batch

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOL = {"float32": 4e-5, "bfloat16": 2.5e-2}
KTOL = {torch.float32: 1e-5, torch.bfloat16: 1.2e-2}


def kernels(dtype):
    from spite_b200.kernels.cuda import CudaKernels
    return CudaKernels(dtype, DEV)


def step_batch(counts, slots, first=False):
    segs, off = [], 0
    for s, n in enumerate(counts):
        segs.append(Segment(s, slots[s], 0, n, off, first))
        off += n
    return build_step_batch(segs, [[0] * n for n in counts], [[] for _ in counts], [[[0]] * len(counts)], DEV), off


def gen(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------------------- the scans
def state_space_loops(q, k, v, step, a_log, dt_bias, skip, S):
    """One head: (outputs [T, vdim], S [dim, vdim])."""
    out = torch.zeros(v.shape, dtype=torch.float64)
    for t in range(q.shape[0]):
        z = float(step[t]) + dt_bias
        dt = max(z, 0.0) + math.log1p(math.exp(-abs(z)))
        S = math.exp(-math.exp(a_log) * dt) * S + dt * torch.outer(k[t], v[t])
        out[t] = S.T @ q[t] + skip * v[t]
    return out, S


def decay_loops(r, k, v, z, w0, u, S):
    out = torch.zeros(v.shape, dtype=torch.float64)
    for t in range(r.shape[0]):
        out[t] = (S + torch.outer(u * k[t], v[t])).T @ r[t]
        S = torch.exp(-torch.exp(z[t] + w0))[:, None] * S + torch.outer(k[t], v[t])
    return out, S


# (heads, kv heads, dim, vdim, segments as token counts of three steps): whole 16-byte groups and not, one column, sizes
# that fill no warp, every shape of the kernel, more than one batch of tokens, exact multiples of a batch
SCAN_CASES = [
    (4, 1, 64, 64, [(19, 1, 8), (1, 1, 1), (40, 2, 3)]),
    (6, 3, 18, 20, [(9, 1, 1), (1, 16, 2), (2, 1, 30)]),
    (3, 3, 10, 10, [(17, 3, 1)]),
    (1, 1, 1, 1, [(5, 1, 2), (1, 1, 1)]),
    (2, 1, 128, 70, [(24, 1, 1), (3, 1, 9)]),
    (2, 2, 136, 136, [(11, 1, 2)]),
    (3, 1, 200, 36, [(8, 8, 1), (1, 1, 7)]),
    (1, 1, 512, 12, [(10, 1, 1)]),
    (2, 2, 33, 33, [(12, 1, 5)]),
]


@pytest.mark.parametrize("kind", ["state space", "decay"])
@pytest.mark.parametrize("case", range(len(SCAN_CASES)))
def test_scans_carried_from_step_to_step(kind, case):
    """Three steps over the same slots, dealt out of order, beside slots that hold leftovers: outputs and matrices are the
    loops', and nothing else in any slot is touched."""
    heads, kvh, dim, vdim, segs = SCAN_CASES[case]
    if kind == "decay":
        kvh = heads
    ks = kernels(torch.float32)
    g = gen(100 + case)
    rnd = lambda *s: torch.randn(s, generator=g)
    n_slots, per = len(segs) + 2, ks.scan_state_size(dim, vdim)
    offset = 8
    state = rnd(n_slots, offset + heads * per + 12).to(DEV)
    slots = torch.randperm(n_slots, generator=g)[:len(segs)].tolist()
    state[torch.tensor(slots)] = 0.0
    start = state.cpu().clone()
    head = dict(a_log=rnd(heads) - 1.0, dt_bias=rnd(heads), skip=rnd(heads))
    w0, u = rnd(heads * dim) - 1.0, rnd(heads * dim)
    Ss = {s: [torch.zeros(dim, vdim, dtype=torch.float64) for _ in range(heads)] for s in range(len(segs))}
    for step in range(3):
        counts = [sg[step] for sg in segs]
        batch, M = step_batch(counts, slots, step == 0)
        x = rnd(M, 4 + 2 * kvh * dim + heads * vdim)             # one tensor, columns from 4 on: q, k, v
        cq, ck, cv = 4, 4 + kvh * dim, 4 + 2 * kvh * dim
        st, z = rnd(M, heads + 3), rnd(M, heads * dim)
        out = torch.full((M, heads * vdim), 7.0, device=DEV)
        xd = x.to(DEV)
        if kind == "state space":
            ks.state_space_scan((xd, cq), (xd, ck), (xd, cv), (st.to(DEV), 2), out, batch, state, heads=heads, kv_heads=kvh, dim=dim,
                                vdim=vdim, state_offset=offset, **{n: t.to(DEV) for n, t in head.items()})
        else:
            wd = z.to(DEV)
            ks.decay_scan((xd, cq), (xd, ck), (xd, cv), wd, out, batch, state, heads=heads, dim=dim, vdim=vdim, w0=w0.to(DEV),
                          u=u.to(DEV), state_offset=offset)
            close(wd, torch.exp(-torch.exp(z.double() + w0.double())), 1e-6, "decays")
        ref = torch.zeros(M, heads * vdim, dtype=torch.float64)
        X, off = x.double(), 0
        for s, n in enumerate(counts):
            for a in range(heads):
                b = a // (heads // kvh)
                q, k = (X[off:off + n, c + b * dim:c + (b + 1) * dim] for c in (cq, ck))
                v = X[off:off + n, cv + a * vdim:cv + (a + 1) * vdim]
                if kind == "state space":
                    o, Ss[s][a] = state_space_loops(q, k, v, st[off:off + n, 2 + a], float(head["a_log"][a]), float(head["dt_bias"][a]),
                                                    float(head["skip"][a]), Ss[s][a])
                else:
                    c = slice(a * dim, (a + 1) * dim)
                    o, Ss[s][a] = decay_loops(q, k, v, z[off:off + n, c].double(), w0[c].double(), u[c].double(), Ss[s][a])
                ref[off:off + n, a * vdim:(a + 1) * vdim] = o
            off += n
        close(out, ref, 5e-6, f"{kind} scan, step {step}")
    got = state.cpu()
    dim4 = -(-dim // 4) * 4
    for s in range(len(segs)):
        mine = got[slots[s], offset:offset + heads * per].view(heads, vdim, dim4)
        close(mine[:, :, :dim].transpose(1, 2), torch.stack(Ss[s]), 5e-6, "matrices")
        assert float(mine[:, :, dim:].abs().sum()) == 0.0        # the padding stays zero
    keep = torch.ones_like(got, dtype=torch.bool)
    keep[torch.tensor(slots), offset:offset + heads * per] = False
    assert torch.equal(got[keep], start[keep])


@pytest.mark.parametrize("kind", ["state space", "decay"])
def test_a_far_token_is_read_back_in_every_cut(kind):
    """One token writes a strong key at position 2, 700 tokens of weak ones follow with next to no decay, the last query asks
    for it: in one prompt, in portions and one by one, bit for bit the same."""
    heads, dim, vdim, T = 2, 48, 32, 700
    ks = kernels(torch.float32)
    g = gen(5)
    q, k, v = (torch.randn((T, heads * n), generator=g) * s for n, s in ((dim, 0.01), (dim, 0.01), (vdim, 1.0)))
    k[2, :dim] = torch.randn(dim, generator=g)
    q[-1, :dim] = k[2, :dim]
    results = []
    for cut in ([T], [300, 2, 7, 391], [690] + [1] * 10):
        state = torch.zeros((1, heads * ks.scan_state_size(dim, vdim)), device=DEV)
        outs, at = [], 0
        for n in cut:
            batch, _ = step_batch([n], [0])
            part = [t[at:at + n].contiguous().to(DEV) for t in (q, k, v)]
            out = torch.empty((n, heads * vdim), device=DEV)
            if kind == "state space":
                z = torch.zeros(heads, device=DEV)
                ks.state_space_scan((part[0], 0), (part[1], 0), (part[2], 0), (torch.zeros((n, heads), device=DEV), 0), out, batch, state,
                                    heads=heads, kv_heads=heads, dim=dim, vdim=vdim, a_log=z - 9.0, dt_bias=z, skip=z)
            else:
                z = torch.zeros(heads * dim, device=DEV)
                ks.decay_scan((part[0], 0), (part[1], 0), (part[2], 0), torch.full((n, heads * dim), -9.0, device=DEV), out, batch, state,
                              heads=heads, dim=dim, vdim=vdim, w0=z, u=z)
            outs.append(out.cpu())
            at += n
        results.append((torch.cat(outs), state.cpu()))
    for o, st in results[1:]:
        assert torch.equal(o, results[0][0]) and torch.equal(st, results[0][1])
    o, v2 = results[0][0][-1, :vdim], v[2, :vdim]
    assert float(torch.nn.functional.cosine_similarity(o, v2, dim=0)) > 0.95      # the far value, hardly disturbed


def test_padding_rows_of_a_captured_step_move_no_state():
    """A captured decode step pads its rows with copies of its first row, slot included: the slot is renewed once by the scans
    and the token shift, and the copies' rows do not reach the cache."""
    ks = kernels(torch.float32)
    g = gen(9)
    heads, dim, d = 2, 16, 24
    per = heads * ks.scan_state_size(dim, dim)
    batch1, _ = step_batch([1, 1], [2, 0])
    batch, M = step_batch([1, 1, 1, 1], [2, 0, 2, 2])
    x = torch.randn((2, 3 * heads * dim), generator=g)
    x4 = torch.cat([x, torch.randn((2, x.shape[1]), generator=g)])          # (behind a recurrent layer a copy's row is another)
    state = torch.randn((3, per + d), generator=g)
    z, w = torch.zeros(heads * dim, device=DEV), torch.randn((2, heads * dim), generator=g)
    mu = torch.rand((2, d), generator=g).to(DEV)
    h = torch.randn((4, d), generator=g)
    got = []
    for b, n, xs in ((batch1, 2, x), (batch, 4, x4)):
        st = state.to(DEV)
        xd, out = xs.to(DEV), torch.empty((n, heads * dim), device=DEV)
        ks.decay_scan((xd, 0), (xd, heads * dim), (xd, 2 * heads * dim), torch.cat([w, w])[:n].to(DEV), out, b, st, heads=heads, dim=dim,
                      vdim=dim, w0=z, u=z)
        mixes = torch.empty((2, n, d), device=DEV)
        ks.token_shift(h[:n].to(DEV), mu, mixes, b, st, state_offset=per)
        got.append((out[:2].cpu(), mixes[:, :2].cpu(), st.cpu()))
        assert bool(torch.isfinite(out).all())
    assert all(torch.equal(a, b) for a, b in zip(*got))
    # the prepare kernel: rows 2 and 3 stand at the first row's position in the first row's page and append nothing
    nq, hd, P = 2, 16, 16
    segs = [Segment(i, 0, 5, 1, i, False) for i in range(3)]
    rows = build_step_batch(segs, [[0]] * 3, [[]] * 3, [[[4], [1], [4]]], DEV)
    kv = torch.zeros((2, 6, 1, P, hd), device=DEV)
    qkv = torch.randn((3, (nq + 2) * hd), generator=g).to(DEV)
    q = torch.empty((3, nq * hd), device=DEV)
    ks.qk_prepare(qkv, q, rows, LayerCache(0, kv, None, P, True), num_heads=nq, rotation=None, qk_norm=None, temperature=None)
    assert torch.equal(kv[0, 4, 0, 5], qkv[0, nq * hd:(nq + 1) * hd]) and torch.equal(kv[1, 4, 0, 5], qkv[0, (nq + 1) * hd:])
    assert torch.equal(kv[0, 1, 0, 5], qkv[1, nq * hd:(nq + 1) * hd])


# ---------------------------------------------------------------------------- token shift, convolution bias, gated norm, streams
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [72, 130, 33, 2048])
def test_token_shift_carried_from_step_to_step(dtype, d):
    ks = kernels(dtype)
    g = gen(d)
    segs, slots, offset, n = [(7, 1, 2), (1, 1, 1), (2, 9, 1)], [3, 0, 2], 5, 5
    state = torch.randn((4, offset + d + 2), generator=g).to(DEV)
    state[torch.tensor(slots)] = 0.0
    start = state.cpu().clone()
    mu = torch.rand((n, d), generator=g)
    last = [torch.zeros(d, dtype=torch.float64) for _ in segs]
    for step in range(3):
        counts = [s[step] for s in segs]
        batch, M = step_batch(counts, slots, step == 0)
        x = torch.randn((M, d), generator=g).to(dtype)
        out = torch.empty((n, M, d), dtype=dtype, device=DEV)
        offs = torch.empty(n + 1, dtype=torch.int32, device=DEV)
        ks.token_shift(x.to(DEV), mu.to(DEV), out, batch, state, state_offset=offset, offsets_out=offs)
        assert offs.tolist() == [i * M for i in range(n + 1)]
        ref, off = torch.zeros(n, M, d, dtype=torch.float64), 0
        for s, c in enumerate(counts):
            for i in range(c):
                cur = x[off + i].double()
                ref[:, off + i] = cur + (last[s] - cur) * mu.double()
                last[s] = cur
            off += c
        close(out, ref, 1e-6 if dtype == torch.float32 else 8e-3, f"token shift, step {step}")
    got = state.cpu()
    for s, slot in enumerate(slots):
        assert torch.equal(got[slot, offset:offset + d].double(), last[s])
    got[torch.tensor(slots), offset:offset + d] = start[torch.tensor(slots), offset:offset + d]
    assert torch.equal(got, start)


@pytest.mark.parametrize("taps,channels", [(1, 40), (4, 130), (8, 7)])
def test_convolution_with_a_bias(taps, channels):
    ks = kernels(torch.float32)
    g = gen(taps)
    state = torch.zeros((2, max(1, (taps - 1) * channels)), device=DEV)
    w, b = torch.randn((channels, taps), generator=g), torch.randn(channels, generator=g)
    x = torch.randn((30, channels + 6), generator=g)
    outs = []
    for lo, hi in ((0, 19), (19, 20), (20, 30)):
        batch, M = step_batch([hi - lo], [1], lo == 0)
        out = torch.empty((M, channels), device=DEV)
        ks.short_conv(x[lo:hi].contiguous().to(DEV), w.to(DEV), out, batch, state, channels=channels, activation="silu", bias=b.to(DEV))
        outs.append(out.cpu())
    pad = torch.cat([torch.zeros(taps - 1, channels), x[:, :channels]]).double()
    y = sum(pad[j:j + 30] * w[:, j].double() for j in range(taps)) + b.double()
    close(torch.cat(outs), y * torch.sigmoid(y), 2e-6, "convolution with a bias")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,size", [(1, 36), (4, 30), (3, 7), (2, 1024), (1, 9000), (5, 1)])
def test_gate_before_a_norm_in_equal_parts(dtype, groups, size):
    ks = kernels(dtype)
    g = gen(size)
    M, n, eps = 5, groups * size, 1e-3
    x, z, gain = torch.randn((M, n), generator=g), torch.randn((M, n + 9), generator=g), torch.randn(n, generator=g)
    x[0, :size] *= 1e-3                                           # (a part whose mean square the epsilon outweighs)
    out = torch.empty((M, n), dtype=dtype, device=DEV)
    ks.gate_group_norm(x.to(DEV), z.to(DEV), gain.to(DEV), out, groups=groups, eps=eps, z_column=4)
    v = x.double() * torch.nn.functional.silu(z[:, 4:4 + n].double())
    v = v.view(M, groups, size)
    ref = (v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)).view(M, n) * gain.double()
    close(out, ref, 2e-6 if dtype == torch.float32 else 8e-3, "gated norm")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,d", [(1, 40), (2, 72), (3, 130), (4, 2048), (5, 48), (7, 33), (4, 20000)])
def test_streams(dtype, n, d):
    """A sublayer's output laid in (with bias and scale), all streams from the old ones; the next sublayer's normed input; the
    last read of some rows alone, which stores nothing; the plain sum."""
    ks = kernels(dtype)
    g = gen(n * d)
    rnd = lambda *s: torch.randn(s, generator=g)
    M, eps = 6, 1e-4
    x, y, bias, scale, mix, wo, wi, gain = rnd(M, n, d), rnd(M, d), rnd(d), rnd(d), rnd(n, n), rnd(n), rnd(n), rnd(d)
    dev = lambda t: t.to(DEV)
    new = torch.einsum("st,msd->mtd", mix.double(), x.double()) + wo.double()[None, :, None] * ((y + 0.0).double() + bias.double())[:, None] * scale.double()
    u = torch.einsum("s,msd->md", wi.double(), new)
    normed = u / torch.sqrt(u.pow(2).mean(-1, keepdim=True) + eps) * gain.double()
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    xd, out = dev(x), torch.empty((M, d), dtype=dtype, device=DEV)
    args = dict(y=dev(y), bias=dev(bias), scale=dev(scale), mix=dev(mix), w_out=dev(wo))
    ks.streams(xd, **args, w_in=dev(wi), gain=dev(gain), eps=eps, next_out=out)
    close(xd, new, 3e-6, "streams"); close(out, normed, tol, "next input")
    xd = dev(x)
    ks.streams(xd, **args)                                        # laid in, nothing read
    close(xd, new, 3e-6, "streams")
    rows = torch.tensor([5, 0, 5], dtype=torch.int32)
    xd, out = dev(x), torch.empty((3, d), dtype=dtype, device=DEV)
    ks.streams(xd, **args, w_in=dev(wi), gain=dev(gain), eps=eps, next_out=out, rows=dev(rows), write_back=False)
    close(out, normed[rows.long()], tol, "last read")
    assert torch.equal(xd.cpu(), x)
    total = torch.empty((M, d), device=DEV)
    ks.streams(xd, w_in=torch.ones(n, device=DEV), next_out=total)
    close(total, x.double().sum(1), 1e-6, "sum of the streams")
    e = torch.empty((4, n, 16), device=DEV)
    table = rnd(9, 16).to(dtype)
    ks.embed(dev(table), torch.tensor([3, 8, 0, 3], dtype=torch.int32, device=DEV), e, copies=n)
    assert torch.equal(e.cpu(), table[[3, 8, 0, 3]].float()[:, None].expand(4, n, 16))


# ---------------------------------------------------------------------------- rotated values, heads turned back
def rotation_of(size, base, pairing="halves"):
    f = torch.tensor([base ** (-2.0 * i / size) for i in range(size // 2)], dtype=torch.float64)
    low = (f - f.float().double()).float()
    return f, Rotation(f.float().to(DEV), pairing, size, inv_freq_low=low.to(DEV))


def turned(v, pos, f, pairing, sign=1.0):
    """v [tokens, heads, size] in float64."""
    n = f.numel()
    a = sign * pos.double()[:, None] * f[None]
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    i0, i1 = (slice(0, n), slice(n, 2 * n)) if pairing == "halves" else (slice(0, 2 * n, 2), slice(1, 2 * n, 2))
    out = v.double().clone()
    out[..., i0], out[..., i1] = v[..., i0].double() * c - v[..., i1].double() * s, v[..., i1].double() * c + v[..., i0].double() * s
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,hd,vd,pairing", [(4, 2, 24, 16, "halves"), (3, 3, 32, 30, "neighbours"), (2, 1, 128, 96, "halves"),
                                                  (6, 2, 64, 64, "halves"), (1, 1, 256, 256, "halves"), (2, 2, 8, 2, "halves")])
def test_values_are_cached_turned_and_heads_turned_back(dtype, nq, nkv, hd, vd, pairing):
    ks = kernels(dtype)
    g = gen(hd + vd)
    P = 16
    specs = [(0, 20), (37, 3), (100000, 1)]
    segs, tables, off = [], [], 0
    for s, (start, n) in enumerate(specs):
        segs.append(Segment(s, s, start, n, off, start == 0))
        off += n
        tables.append([-1] * (start // P) + list(range(3 * s, 3 * s + (start + n - 1) // P - start // P + 1)))
    M = off
    batch = build_step_batch(segs, [[0] * n for _, n in specs], [[]] * 3, [tables], DEV)
    f, rot = rotation_of(vd, 500.0, pairing)
    fk, rk = rotation_of(2 * (hd // 4), 100.0)
    x = torch.randn((M, (nq + 2 * nkv) * hd), generator=g).to(dtype)
    kv = torch.zeros((2, 9, nkv, P, hd), dtype=dtype, device=DEV)
    q = torch.empty((M, nq * hd), dtype=dtype, device=DEV)
    ks.qk_prepare(x.to(DEV), q, batch, LayerCache(0, kv, None, P, True), num_heads=nq, rotation=rk, qk_norm=None, temperature=None,
                  value_rotation=rot)
    pos = torch.cat([torch.arange(a, a + n) for a, n in specs])
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    want_v = turned(x.view(M, -1, hd)[:, nq + nkv:], pos, f, pairing)
    want_k = turned(x.view(M, -1, hd)[:, nq:nq + nkv], pos, fk, "halves")
    got_k, got_v = torch.zeros(M, nkv, hd), torch.zeros(M, nkv, hd)
    t = 0
    for s, (start, n) in enumerate(specs):
        for p in range(start, start + n):
            got_k[t], got_v[t] = kv[0, tables[s][p // P], :, p % P].float().cpu(), kv[1, tables[s][p // P], :, p % P].float().cpu()
            t += 1
    close(got_v, want_v, tol, "cached values"); close(got_k, want_k, tol, "cached keys")     # (position 100,000 included)
    o = torch.randn((M, nq * hd), generator=g).to(dtype)
    out = torch.full((M, nq * vd + 10), 3.0, dtype=dtype, device=DEV)
    ks.turn_heads(o.to(DEV), out, batch, heads=nq, size=vd, rotation=rot, scale=0.8, out_column=6)
    ref = 0.8 * turned(o.view(M, nq, hd)[..., :vd], pos, f, pairing, sign=-1.0).reshape(M, nq * vd)
    close(out[:, 6:6 + nq * vd], ref, tol, "heads turned back")
    assert bool((out[:, :6] == 3.0).all()) and bool((out[:, 6 + nq * vd:] == 3.0).all())
    ks.turn_heads(o.to(DEV), out, batch, heads=nq, size=vd, out_column=0)
    assert torch.equal(out[:, :nq * vd].cpu(), o.view(M, nq, hd)[..., :vd].reshape(M, nq * vd))


# ---------------------------------------------------------------------------- products
@pytest.mark.parametrize("dtype,M,N,K,library", [
    (torch.float32, 5, 70, 50, "gemm_simt"), (torch.float32, 130, 96, 72, "gemm_simt"), (torch.bfloat16, 3, 200, 128, "gemm_stream"),
    (torch.bfloat16, 9, 520, 1024, "gemm_stream"), (torch.bfloat16, 5, 72, 160, "gemm_skinny"), (torch.bfloat16, 40, 150, 72, "gemm_tc"),
    (torch.bfloat16, 130, 257, 64, "gemm_tc"), (torch.bfloat16, 300, 264, 200, "gemm_tc_pair"), (torch.bfloat16, 70, 33, 50, "gemm_simt")])
@pytest.mark.parametrize("activation", ["xielu", "tanh", None])
def test_bias_and_activation_in_every_product_kernel(dtype, M, N, K, library, activation):
    ks = kernels(dtype)
    g = gen(M + N)
    x, w = torch.randn((M, K), generator=g).to(dtype), (torch.randn((N, K), generator=g) * 1.5 / K ** 0.5).to(dtype)
    b = torch.randn(N, generator=g)
    out = torch.empty((M, N), dtype=dtype, device=DEV)
    ap, an = 1.3, 0.9
    more = {"act_params": (ap, an)} if activation == "xielu" else {}
    ks.linear(x.to(DEV), w.to(DEV), out, activation=activation, bias=b.to(DEV), **more)
    assert ks.launches_by_library[library] == 1, dict(ks.launches_by_library)
    z = x.double() @ w.double().T + b.double()
    n = torch.clamp(z, max=0)
    ref = torch.tanh(z) if activation == "tanh" else z if activation is None else \
        torch.where(z > 0, ap * z * z, an * (torch.expm1(n) - n)) + z / 2
    close(out, ref, 3e-6 if dtype == torch.float32 else 8e-3, f"bias and {activation}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G,M,N,K", [(4, 1, 136, 256), (4, 3, 72, 40), (4, 8, 256, 128), (4, 33, 96, 72), (2, 300, 128, 64), (4, 600, 64, 128), (3, 5, 33, 50)])
def test_one_product_per_group(dtype, G, M, N, K):
    ks = kernels(dtype)
    g = gen(G * M)
    x, w = torch.randn((G, M, K), generator=g).to(dtype), torch.randn((G, N, K), generator=g).to(dtype)
    out = torch.empty((G, M, N), device=DEV)
    ks.batched_linear(x.to(DEV), w.to(DEV), torch.arange(G + 1, dtype=torch.int32, device=DEV) * M, out)
    close(out, torch.einsum("gmk,gnk->gmn", x.double(), w.double()), 3e-6, "one product per group")      # (float32 sums in both sets)


# ---------------------------------------------------------------------------- the left mixer around a window's edge
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hd,window", [(64, 100), (24, 20), (128, 64), (96, 33)])
def test_keys_just_inside_and_just_outside_the_window(dtype, hd, window):
    """A query that is aligned with the oldest key it may see, and with the one just before it, in a prompt and decoded: the
    value of the first comes out (turned by its distance), that of the second does not."""
    from spite_b200.config import PartSpec
    from spite_b200.parts import BuildContext, build_part
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    ks = kernels(tdt)
    ctx = BuildContext(kernels=ks, dtype=tdt, device=torch.device(DEV))
    vd, d, T = 16, 64, 2 * window + 9
    mixer = build_part("mixer", PartSpec("paged_attention", {
        "hidden_size": d, "num_heads": 1, "num_kv_heads": 1, "head_dim": hd, "value_dim": vd, "softmax_scale": 1.0,
        "window": ("sliding", window), "position": PartSpec("no_position", {}),
        "value_rotation": PartSpec("rotary_halves", {"rotary_dim": vd, "theta": 100.0, "exact_angles": True})}), ctx)
    # the first dimensions of the input are the query, the next the key, the last the value
    wq, wk, wv = torch.zeros(hd, d), torch.zeros(hd, d), torch.zeros(vd, d)
    for i in range(8):
        wq[i, i], wk[i, 8 + i] = 1.0, 1.0
    wv[:, 32:32 + vd] = torch.eye(vd)
    mixer.bind({"q_proj": wq.to(DEV), "k_proj": wk.to(DEV), "v_proj": wv.to(DEV), "o_proj": torch.eye(d)[:, :vd].contiguous().to(DEV)})
    x = torch.zeros(T, d)
    x[:, 32:32 + vd] = torch.randn((T, vd), generator=gen(window)) * 0.1
    i = T - 2                                                     # asks for i - window + 1, and the last token for the same key: outside
    far = i - window + 1
    x[far, 32:32 + vd] = torch.randn(vd, generator=gen(3))
    x[far, 8], x[i, 0], x[i + 1, 0] = 6.0, 6.0, 6.0
    P = 16
    pages = -(-T // P)
    kv = torch.zeros((2, pages, 1, P, mixer.hd), dtype=tdt, device=DEV)
    xd = x.to(tdt).to(DEV)
    for cut in (T, T - 2):
        h = torch.zeros((T, d), device=DEV)
        kv.zero_()
        for lo, hi in [(0, cut)] + [(t, t + 1) for t in range(cut, T)]:
            batch = build_step_batch([Segment(0, 0, lo, hi - lo, 0, lo == 0)], [[0] * (hi - lo)], [[]], [[list(range(pages))]], DEV)
            part = h[lo:hi].contiguous()
            mixer.forward(xd[lo:hi].contiguous(), part, batch, LayerCache(0, kv, None, P, True), accumulate=False)
            h[lo:hi] = part
        f, _ = rotation_of(vd, 100.0)
        v = x[:, 32:32 + vd].to(tdt).double()
        want = turned(v[far][None, None], torch.tensor([-(i - far)]), f, "halves")[0, 0]
        tol = 1e-4 if dtype == "float32" else 3e-2
        assert float((h[i, :vd].cpu().double() - want).abs().max()) <= tol * float(want.abs().max())
        assert float(h[i + 1, :vd].abs().max()) < 0.3 * float(want.abs().max())       # an average of small values


# ---------------------------------------------------------------------------- the engine
@pytest.fixture(scope="module", params=list(S.CONFIGS))
def folder(request, tmp_path_factory):
    return S.write_model(tmp_path_factory.mktemp(f"zuzadra_{request.param}"), request.param), request.param


@pytest.fixture(scope="module", params=["float32", "bfloat16"])
def setup(request, folder):
    from spite_b200.engine import Model
    path, name = folder
    dtype = request.param
    model = Model.from_folder(path, dtype=dtype, device=DEV)
    vocab = model.plan.vocab_size
    lengths = {"a": 210 if name == "Q" else 97, "b": 40, "c": 37, "d": 66, "e": 1, "f": 21}
    requests = {r: H.random_tokens(vocab, n, i) for i, (r, n) in enumerate(lengths.items())}
    return path, model, requests, TOL[dtype], dtype


def _engine(model, steps, page_size, max_requests=4):
    from spite_b200.engine import Engine
    return Engine(model, cache_tokens=H.max_tokens_of(steps), page_size=page_size, max_requests=max_requests)


def poison_free_pages(engine):
    """Whatever a free page held last is not finite: a kernel that reads a masked key of a reused page shows it."""
    for g, pool in enumerate(engine.cache.pools):
        if pool._free:
            engine.storage.kv[g][:, :, torch.tensor(pool._free, device=DEV)] = float("nan")


def test_every_cut_gives_the_logits_of_the_whole_sequence(setup):
    path, model, requests, tol, dtype = setup
    n_prompt = {r: max(1, len(t) - 9) for r, t in requests.items()}
    cuts = {"whole": (H.steps_whole(requests), 64), "whole, small pages": (H.steps_whole(requests), 16),
            "last 32 decoded": (H.steps_last_decoded(requests, 32), 64),
            "portions": (H.steps_portions(requests, seed=4), 64),
            "portions of 2 and 3": (H.steps_portions(requests, seed=5, sizes=(2, 3)), 16),
            "mixed": (H.steps_mixed(requests, n_prompt, seed=6), 64),
            "mixed, small pages": (H.steps_mixed(requests, n_prompt, seed=7, sizes=(2, 5, 17, 40)), 16)}
    results = {}
    for what, (steps, page) in cuts.items():
        eng = _engine(model, steps, page)
        results[what] = H.run_steps(eng, steps, before_step=poison_free_pages)
        S.compare_with_plain(results[what], path, requests, tol)
        eng.check()
        assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups, what
    if dtype == "float32":
        H.assert_cuts_identical(results)


def test_the_sum_of_the_streams_layer_run_by_layer_run(setup):
    path, model, requests, tol, dtype = setup
    cfg, tensors = S.folder_contents(str(path))
    toks = requests["c"]
    layers = []
    plain.forward(cfg, tensors, toks, torch.float64, taps=layers)
    seen = []
    model.layer_tap = lambda i, h: seen.append(h.double().cpu())
    try:
        steps = H.steps_whole({"c": toks})
        H.run_steps(_engine(model, steps, 64), steps)
    finally:
        model.layer_tap = None
    assert len(seen) == len(layers)
    for i, h in enumerate(seen):
        err = float((h - layers[i]).abs().max()) / float(layers[i].abs().max())
        assert err <= (4e-5 if dtype == "float32" else 5e-2), f"layer run {i}: {err:.3e}"


def test_long_decoding_after_a_short_prompt(setup):
    """Three prompt tokens, then 160 tokens one by one (decode steps replayed from CUDA graphs, pages taken one after
    the other, every window of the configuration crossed while decoding)."""
    path, model, requests, tol, dtype = setup
    reqs = {"long": H.random_tokens(model.plan.vocab_size, 163, 77)}
    steps = H.steps_last_decoded(reqs, 160)
    eng = _engine(model, steps, 16)
    S.compare_with_plain(H.run_steps(eng, steps), path, reqs, tol)
    assert eng.graph_replays > 100


def test_decode_steps_of_many_requests_from_graphs(setup):
    """Eleven requests decode side by side and end one by one: the captured steps' padding rows (copies of the first row, slot
    included; ten, twelve and so on rows serve nine and eleven requests) leave states and caches as they were."""
    path, model, requests, tol, dtype = setup
    reqs = {f"r{i}": H.random_tokens(model.plan.vocab_size, 16 + i, 200 + i) for i in range(11)}
    steps = [{"entries": [{"id": r, "tokens": t[:5], "want": list(range(5))} for r, t in reqs.items()], "end": []}]
    for i in range(5, 26):
        live = [(r, t) for r, t in reqs.items() if i < len(t)]
        steps.append({"entries": [{"id": r, "tokens": [t[i]], "want": [0]} for r, t in live],
                      "end": [r for r, t in live if i == len(t) - 1]})
    for i, s in enumerate(steps):
        s["step"] = i
    eng = _engine(model, steps, 16, max_requests=11)
    S.compare_with_plain(H.run_steps(eng, steps), path, reqs, tol)
    assert eng.graph_replays > 8


def test_greedy_generation_through_the_entry_point(setup):
    """`LLM.generate` (scheduler, sampler, engine): the tokens are the plain implementation's argmax at every
    step where its best two logits are not within rounding of each other."""
    from spite_b200 import LLM
    path, model, requests, tol, dtype = setup
    cfg, tensors = S.folder_contents(str(path))
    prompts = [requests["b"][:30], requests["c"][:7], requests["f"][:2], requests["d"][:50]]
    llm = LLM(model, cache_tokens=4 * 128, page_size=16, max_requests=3, max_batch_tokens=24)
    outs = llm.generate(prompts, max_tokens=12, temperature=0.0)
    compared = 0
    for prompt, out in zip(prompts, outs):
        assert len(out) == 12
        rows = plain.forward(cfg, tensors, list(prompt) + list(out))             # (the engine's own sequence)
        for i, tok in enumerate(out):
            row = rows[len(prompt) - 1 + i]
            top2 = torch.topk(row, 2).values
            if float(top2[0] - top2[1]) > 2 * max(tol, 5e-2 if dtype == "bfloat16" else 0) * float(row.abs().max()):
                assert tok == int(torch.argmax(row)), f"after {len(prompt) + i} tokens"
                compared += 1
    assert compared >= (12 if dtype == "float32" else 4)


def test_the_layers_side_by_side_or_one_after_the_other(folder):
    """The right mixer on a side stream or behind the left one: the same bits."""
    from spite_b200.engine import Model
    path, name = folder
    model = Model.from_folder(path, dtype="float32", device=DEV)
    toks = H.random_tokens(model.plan.vocab_size, 50, 8)
    results = []
    for beside in (True, False):
        for b in model.blocks:
            if b.mixer.kind == "parallel_mixers":
                b.mixer.side_by_side = beside
        steps = H.steps_last_decoded({"a": toks}, 10)
        results.append(H.run_steps(_engine(model, steps, 16), steps))
    assert all(torch.equal(results[0][k], results[1][k]) for k in results[0])


def test_trace_replay_program(folder, tmp_path):
    """`bin/trace_run` as a program: a mixed schedule in, logits files out, equal to the plain implementation."""
    import subprocess, sys
    import numpy as np
    from pathlib import Path
    path, name = folder
    if name not in ("P", "Q"):
        pytest.skip("two configurations run as programs")
    vocab = json.loads((path / "config.json").read_text())["vocab"]
    requests = {r: H.random_tokens(vocab, n, 90 + i) for i, (r, n) in enumerate({"a": 70, "b": 33, "c": 5}.items())}
    steps = H.steps_mixed(requests, {r: len(t) - 4 for r, t in requests.items()}, seed=9)
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(path), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", str(H.max_tokens_of(steps))],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    pos, got = {}, {}
    for s in steps:
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab)
        i = 0
        for e in s["entries"]:
            base = pos.get(e["id"], 0)
            for w in e["want"]:
                got[(e["id"], base + w)] = torch.from_numpy(rows[i].copy())
                i += 1
            pos[e["id"]] = base + len(e["tokens"])
        assert i == rows.shape[0]
    S.compare_with_plain(got, path, requests, 4e-5)


def test_the_command_line_runs_a_zuzadra_folder(tmp_path):
    """`spite random`, `spite run` (greedy, float32: the plain implementation's tokens) and `spite bench`."""
    import subprocess, sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    spite = lambda *a: subprocess.run([sys.executable, str(root / "bin" / "spite")] + [str(x) for x in a],
                                      capture_output=True, text=True, timeout=900)
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(S.CONFIG_P))
    model = tmp_path / "model"
    assert spite("random", "--config", cfg_file, "--out", model, "--seed", 3, "--std", 0.3).returncode == 0
    cfg, W = plain.load_folder(model)
    prompt = H.random_tokens(211, 17, 2)
    proc = spite("run", "-m", model, "-p", " ".join(map(str, prompt)), "--max-tokens", 6, "--temperature", 0,
                 "--dtype", "fp32", "--page-size", 16, "--num-pages", 8)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [int(t) for t in proc.stdout.split()] == S.generate_greedy(cfg, W, prompt, 6)
    proc = spite("bench", "-m", model, "--n-prompt", 40, "--n-tokens", 12, "--n-runs", 2, "--json", "--dtype", "bf16")
    assert proc.returncode == 0, proc.stderr[-2000:]
    report = json.loads(proc.stdout)
    assert report["decode_tps"] > 0 and report["prefill_tps"] > 0
