"""Fozutar on the GPU.  First every new mechanism alone against loops written here from its equation, in float64 (gated linear
attention in prompts, portions and decoded tokens with a far token and slots used again, scores with a number by distance in
every attention kernel with keys just inside and outside a chunk, values that are the projected keys, gelu-gated products in
every product kernel, a biased router, what is added between two passes); then the engine in float32 and bfloat16 against the
plain implementation in every cut (whole, token by token, portions down to two tokens, mixed batches in a pool whose pages and
slots are used again, free pages poisoned), layer run by layer run, long decoding, captured steps with padding rows, greedy
generation through `LLM.generate`, `bin/trace_run` and the command line."""
import json
import math

import pytest
import torch

import fozutar_helpers as S
import helpers as H
import plain_fozutar as plain
from reference_kernels import TorchReferenceKernels
from spite_b200.cache import LayerCache, Window
from spite_b200.engine.batch import Segment, build_step_batch
from spite_b200.kernels.api import DistanceBias
from spite_b200.parts import QkNorm
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


# ---------------------------------------------------------------------------- gated linear attention
def gla_loops(q, k, v, alpha, scale, S):
    """One head: (outputs [T, vdim], S [dim, vdim]), the read-out after the write."""
    out = torch.zeros(v.shape, dtype=torch.float64)
    for t in range(q.shape[0]):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out[t] = scale * (S.T @ q[t])
    return out, S


# (heads, dim, vdim, rank, tau, segments as token counts of three steps): whole 16-byte groups and not, one element, every shape
# of the kernel, more than one batch of tokens, inner sizes of the decay of one and of more than a piece
GLA_CASES = [
    (4, 64, 64, 16, 16.0, [(19, 1, 8), (1, 1, 1), (40, 2, 3)]),
    (3, 18, 20, 5, 7.0, [(9, 1, 1), (1, 16, 2), (2, 1, 30)]),
    (1, 1, 1, 1, 1.0, [(5, 1, 2), (1, 1, 1)]),
    (2, 128, 70, 64, 20.0, [(24, 1, 1), (3, 1, 9)]),
    (2, 136, 136, 65, 3.0, [(11, 1, 2)]),
    (1, 512, 12, 130, 16.0, [(10, 1, 1)]),
    (5, 33, 7, 8, 30.0, [(12, 1, 5), (8, 8, 8)]),
]


@pytest.mark.parametrize("case", range(len(GLA_CASES)))
def test_gated_linear_attention_carried_from_step_to_step(case):
    """Three steps over the same slots, dealt out of order, beside slots that hold leftovers: outputs, decays and matrices are
    the loops', and nothing else in any slot is touched."""
    heads, dim, vdim, rank, tau, segs = GLA_CASES[case]
    ks = kernels(torch.float32)
    g = gen(100 + case)
    rnd = lambda *s: torch.randn(s, generator=g)
    n_slots, per = len(segs) + 2, ks.scan_state_size(dim, vdim)
    offset = 8
    state = rnd(n_slots, offset + heads * per + 12).to(DEV)
    slots = torch.randperm(n_slots, generator=g)[:len(segs)].tolist()
    state[torch.tensor(slots)] = 0.0
    start = state.cpu().clone()
    a2, b = rnd(rank, heads * dim) * 2.0 / rank ** 0.5, rnd(heads * dim) * 2.0
    scale = dim ** -0.5
    Ss = {s: [torch.zeros(dim, vdim, dtype=torch.float64) for _ in range(heads)] for s in range(len(segs))}
    for step in range(3):
        counts = [sg[step] for sg in segs]
        batch, M = step_batch(counts, slots, step == 0)
        cq, ck, cv, ca = 4, 4 + heads * dim, 4 + 2 * heads * dim, 5 + 2 * heads * dim + heads * vdim
        x = rnd(M, ca + rank + 2)
        out, w = torch.full((M, heads * vdim), 7.0, device=DEV), torch.empty((M, heads * dim), device=DEV)
        xd = x.to(DEV)
        ks.gated_linear_scan((xd, cq), (xd, ck), (xd, cv), (xd, ca), w, out, batch, state, heads=heads, dim=dim, vdim=vdim,
                             a2=a2.to(DEV), a2_bias=b.to(DEV), tau=tau, q_scale=scale, state_offset=offset)
        X = x.double()
        alpha = torch.sigmoid(X[:, ca:ca + rank] @ a2.double() + b.double()) ** (1.0 / tau)
        close(w, alpha, 2e-6, "decays")
        ref, off = torch.zeros(M, heads * vdim, dtype=torch.float64), 0
        for s, n in enumerate(counts):
            for a in range(heads):
                c = slice(a * dim, (a + 1) * dim)
                q, k = (X[off:off + n, col + a * dim:col + (a + 1) * dim] for col in (cq, ck))
                ref[off:off + n, a * vdim:(a + 1) * vdim], Ss[s][a] = gla_loops(
                    q, k, X[off:off + n, cv + a * vdim:cv + (a + 1) * vdim], alpha[off:off + n, c], scale, Ss[s][a])
            off += n
        close(out, ref, 5e-6, f"step {step}")
    got = state.cpu()
    dim4 = -(-dim // 4) * 4
    for s in range(len(segs)):
        mine = got[slots[s], offset:offset + heads * per].view(heads, vdim, dim4)
        close(mine[:, :, :dim].transpose(1, 2), torch.stack(Ss[s]), 5e-6, "matrices")
        assert float(mine[:, :, dim:].abs().sum()) == 0.0        # the padding stays zero
    keep = torch.ones_like(got, dtype=torch.bool)
    keep[torch.tensor(slots), offset:offset + heads * per] = False
    assert torch.equal(got[keep], start[keep])


def test_a_far_token_is_read_back_in_every_cut_and_padding_rows_move_nothing():
    """One token writes a strong key at position 2, 700 tokens of weak ones follow with next to no decay, the last query asks
    for it: in one prompt, in portions and one by one, bit for bit the same.  Then a captured step's padding rows (copies of the
    first row's slot) renew that slot once."""
    heads, dim, vdim, T = 2, 48, 32, 700
    ks = kernels(torch.float32)
    g = gen(5)
    x = torch.randn((T, heads * (2 * dim + vdim) + 3), generator=g)
    x[:, :2 * heads * dim] *= 0.01
    ck, cv, ca = heads * dim, 2 * heads * dim, 2 * heads * dim + heads * vdim
    x[2, ck:ck + dim] = torch.randn(dim, generator=g)
    x[-1, :dim] = x[2, ck:ck + dim]
    a2, b = torch.zeros((3, heads * dim), device=DEV), torch.full((heads * dim,), 12.0, device=DEV)

    def run(rows, batch, state):
        xd = rows.contiguous().to(DEV)
        out = torch.empty((rows.shape[0], heads * vdim), device=DEV)
        ks.gated_linear_scan((xd, 0), (xd, ck), (xd, cv), (xd, ca), torch.empty((rows.shape[0], heads * dim), device=DEV), out, batch,
                             state, heads=heads, dim=dim, vdim=vdim, a2=a2, a2_bias=b, tau=16.0, q_scale=1.0)
        return out.cpu()
    results = []
    for cut in ([T], [300, 2, 7, 391], [690] + [1] * 10):
        state = torch.zeros((1, heads * ks.scan_state_size(dim, vdim)), device=DEV)
        outs, at = [], 0
        for n in cut:
            outs.append(run(x[at:at + n], step_batch([n], [0])[0], state))
            at += n
        results.append((torch.cat(outs), state.cpu()))
    for o, st in results[1:]:
        assert torch.equal(o, results[0][0]) and torch.equal(st, results[0][1])
    assert float(torch.nn.functional.cosine_similarity(results[0][0][-1, :vdim], x[2, cv:cv + vdim], dim=0)) > 0.95
    state = torch.randn((3, heads * ks.scan_state_size(dim, vdim)), generator=g)
    two, four = state.to(DEV), state.to(DEV)
    a = run(x[:2], step_batch([1, 1], [2, 0])[0], two)
    c = run(x[:4], step_batch([1, 1, 1, 1], [2, 0, 2, 2])[0], four)
    assert torch.equal(a, c[:2]) and torch.equal(two, four) and bool(torch.isfinite(c).all())


# ---------------------------------------------------------------------------- a number by distance, kernel by kernel
def attention_reference(q, k_all, v_all, specs, nq, nkv, scale, window, cap, table, far):
    out = torch.zeros(q.shape[:2] + (v_all[0].shape[-1],), dtype=torch.float64)
    group, off = nq // nkv, 0
    for s, (start, n) in enumerate(specs):
        for t in range(n):
            pos = start + t
            lo = window.lowest_visible(pos)
            number = table[[plain.bucket(pos - j, table.shape[0], far) for j in range(lo, pos + 1)]].double()
            for h in range(nq):
                sc = (k_all[s][lo:pos + 1, h // group].double() @ q[off + t, h].double()) * scale
                if cap is not None:
                    sc = cap * torch.tanh(sc / cap)
                out[off + t, h] = torch.softmax(sc + number[:, h], 0) @ v_all[s][lo:pos + 1, h // group].double()
        off += n
    return out


# (kernel library that must serve the call, dtype, query heads, kv heads, row size, page size, window, cap, (rows, far), segments, a factor
# per key and keys that are the values): tables that end within the first tile, far beyond every key, and between; segments that start in the middle of a chunk; the
# tcgen05 cases have tiles with one number, with many, and row tiles whose keys straddle the table's end
DISTANCE_CASES = [
    ("attention", torch.float32, 5, 1, 24, 16, ("chunk", 50), 3.0, (8, 13), [(0, 1), (0, 60), (130, 1), (99, 3)], True),
    ("attention", torch.bfloat16, 6, 3, 24, 16, ("full", 0), None, (32, 100), [(0, 1), (0, 40), (130, 1), (61, 7)], False),
    ("attention_mma", torch.bfloat16, 4, 2, 48, 16, ("chunk", 200), 4.0, (16, 60), [(0, 1), (199, 1), (200, 1), (398, 3), (1500, 1)], True),
    ("attention_rows", torch.bfloat16, 6, 2, 32, 32, ("sliding", 40), 2.0, (6, 31), [(0, 45), (100, 30), (0, 12), (78, 4)], True),
    ("attention_decode", torch.bfloat16, 8, 2, 64, 64, ("chunk", 900), 6.0, (32, 512), [(0, 1), (63, 1), (899, 1), (900, 1), (3000, 1), (517, 2)], True),
    ("attention_decode", torch.bfloat16, 8, 4, 128, 64, ("chunk", 100), None, (10, 3000), [(99, 1), (100, 1), (299, 1), (250, 1)], False),
    ("attention_tc", torch.bfloat16, 6, 2, 64, 64, ("chunk", 600), 5.0, (32, 128), [(0, 300), (450, 330), (0, 70)], True),
    ("attention_tc", torch.bfloat16, 4, 1, 128, 64, ("full", 0), None, (8, 900), [(0, 140), (900, 64)], False),
    ("attention_tc", torch.bfloat16, 2, 2, 64, 64, ("sliding", 70), 3.0, (4, 3), [(0, 400), (130, 129)], True),
    ("attention", torch.bfloat16, 20, 1, 12, 16, ("chunk", 70), None, (8, 13), [(0, 33), (100, 2)], True),
    ("attention_mma", torch.bfloat16, 2, 1, 64, 16, ("full", 0), None, (2, 2), [(40, 1), (700, 5)], True),
    ("attention_rows", torch.bfloat16, 4, 1, 128, 32, ("chunk", 100), 9.0, (32, 64), [(0, 20), (85, 31)], True),
    ("attention_decode", torch.bfloat16, 4, 2, 128, 128, ("sliding", 333), None, (16, 200), [(1500, 1), (40, 3), (127, 1)], True),
    ("attention_tc", torch.bfloat16, 4, 2, 128, 128, ("chunk", 400), 6.0, (32, 300), [(0, 450), (330, 140)], True),
    ("attention_tc", torch.bfloat16, 16, 1, 64, 64, ("chunk", 250), 8.0, (64, 63 * 64), [(0, 90), (240, 20)], False),
]


@pytest.mark.parametrize("case", range(len(DISTANCE_CASES)))
def test_numbers_by_distance_in_every_attention_kernel(case):
    """Numbers of the size of the scores, different for every head; a last row whose query is aligned with the first key it
    may see, where the key just outside the chunk or window would have taken the row over."""
    library, dtype, nq, nkv, hd, P, win, cap, (rows, far), specs, keys_alone = DISTANCE_CASES[case]
    from spite_b200.parts.position import distance_rows
    ks = kernels(dtype)
    window = Window(*win)
    n_pages = sum(-(-(s + n) // P) for s, n in specs) + 3
    batch, tables = make_batch(specs, P, n_pages, 160 + case, DEV)
    M = batch.n_tokens
    g = gen(161 + case)
    k_all = [torch.randn((s + n, nkv, hd), generator=g).to(dtype) for s, n in specs]
    v_all = k_all if keys_alone else [torch.randn((s + n, nkv, hd), generator=g).to(dtype) for s, n in specs]
    f_all = [torch.rand((s + n, nkv), generator=g) + 0.5 if keys_alone else torch.ones((s + n, nkv)) for s, n in specs]
    q = torch.randn((M, nq, hd), generator=g) * 1.5
    last_pos = specs[-1][0] + specs[-1][1] - 1
    first_seen = window.lowest_visible(last_pos)
    q[M - 1, nq - 1] = k_all[-1][first_seen, nkv - 1].float() * (12.0 / math.sqrt(hd))
    if first_seen > 0:                                       # the key just outside is aligned even better
        k_all[-1][first_seen - 1, nkv - 1] = k_all[-1][first_seen, nkv - 1] * 1.5
    q = q.to(dtype)
    table = torch.randn((rows, nq), generator=g) * 2.0
    length = far + 1 if window.kind == "full" else min(window.size, far + 1)
    bias = DistanceBias.from_rows(table.to(DEV), distance_rows(rows, far, length))
    kv = torch.zeros((2, n_pages, nkv, P, hd), dtype=dtype)
    fill_cache(kv, tables, [(s + n, 0) for s, n in specs], k_all, v_all, P)
    factors = None
    if keys_alone:                                           # what no key is behind may be anything but must not show
        factors = torch.full((n_pages, nkv, P), float("nan"))
        for s, f in enumerate(f_all):
            for p in range(f.shape[0]):
                factors[tables[s][p // P], :, p % P] = f[p]
        kv, factors = kv[:1].contiguous(), factors.to(DEV)
    out = torch.empty((M, nq * hd), dtype=dtype, device=DEV)
    scale = 1.0 / math.sqrt(hd)
    ks.paged_attention(q.reshape(M, nq * hd).to(DEV), out, batch, LayerCache(0, kv.to(DEV), None, P, False, factors),
                       num_heads=nq, window=window, softmax_scale=scale, score_softcap=cap, distance_bias=bias)
    torch.cuda.synchronize()
    assert not ks.errors()
    assert ks.launches_by_library[library] > 0, dict(ks.launches_by_library)
    scaled = [k.double() * f[:, :, None].double() for k, f in zip(k_all, f_all)]
    reference = lambda win, table: attention_reference(q, scaled, v_all, specs, nq, nkv, scale, win, cap, table, far)
    ref = reference(window, table)
    close(out.view(M, nq, hd), ref, KTOL[dtype], f"numbers by distance ({library})")
    assert float((reference(window, table.roll(1, 0)) - ref).abs().max()) > 0.03
    if first_seen > 0:
        assert float((reference(Window("full", 0), table) - ref).abs().max()) > 1e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,kd,hd", [(4, 2, 24, 24), (3, 3, 9, 10), (6, 1, 64, 64), (2, 1, 128, 128), (1, 1, 256, 256)])
def test_values_are_the_projected_keys(dtype, nq, nkv, kd, hd):
    """Rows of q and k heads alone: a key is cached as projected, bias included, and beside it what its norm multiplies it by."""
    ks, ref = kernels(dtype), TorchReferenceKernels(dtype, "cpu")
    P, specs = 16, [(0, 5), (37, 1), (20, 3)]
    n_pages = sum(-(-(s + n) // P) for s, n in specs) + 2
    batch, _ = make_batch(specs, P, n_pages, 31, DEV)
    batch_c, _ = make_batch(specs, P, n_pages, 31, "cpu")
    M, g = batch.n_tokens, gen(32)
    qk, bias = torch.randn((M, nq + nkv, hd), generator=g), torch.randn((nq + nkv, hd), generator=g)
    qk[..., kd:], bias[:, kd:] = 0.0, 0.0
    qk, bias = qk.reshape(M, -1).to(dtype), bias.reshape(-1)
    for norm in (QkNorm(1e-3), None):
        got = []
        for k, dev, b in ((ks, DEV, batch), (ref, "cpu", batch_c)):
            kv, q = torch.zeros((1, n_pages, nkv, P, hd), dtype=dtype, device=dev), torch.empty((M, nq * hd), dtype=dtype, device=dev)
            factors = torch.zeros((n_pages, nkv, P), device=dev)
            k.qk_prepare(qk.to(dev), q, b, LayerCache(0, kv, None, P, True, factors), num_heads=nq, rotation=None, qk_norm=norm,
                         temperature=None, bias=bias.to(dev), norm_dim=kd, values_are_keys=True)
            got.append((q.cpu(), kv.cpu(), factors.cpu()))
        tol = 2e-6 if dtype == torch.float32 else 8e-3
        for a, b, t, what in zip(got[0], got[1], (tol, tol, 1e-6), ("queries", "keys as projected", "factors")):
            close(a, b, t, what)


# ---------------------------------------------------------------------------- products, router, junction
@pytest.mark.parametrize("dtype,M,N,K,library", [
    (torch.float32, 5, 70, 50, "gemm_simt"), (torch.float32, 130, 96, 72, "gemm_simt"), (torch.bfloat16, 3, 200, 128, "gemm_stream"),
    (torch.bfloat16, 9, 520, 1024, "gemm_stream"), (torch.bfloat16, 5, 72, 160, "gemm_skinny"), (torch.bfloat16, 40, 150, 72, "gemm_tc"),
    (torch.bfloat16, 130, 257, 64, "gemm_tc"), (torch.bfloat16, 300, 264, 200, "gemm_tc_pair"), (torch.bfloat16, 70, 33, 50, "gemm_simt")])
def test_gelu_gates_in_every_product_kernel(dtype, M, N, K, library):
    ks = kernels(dtype)
    g = gen(M + N)
    x, w = torch.randn((M, K), generator=g).to(dtype), (torch.randn((2 * N, K), generator=g) * 1.5 / K ** 0.5).to(dtype)
    out, silu = (torch.empty((M, N), dtype=dtype, device=DEV) for _ in range(2))
    ks.linear_swiglu(x.to(DEV), w.to(DEV), out, activation="gelu_tanh")
    assert ks.launches_by_library[library] == 1, dict(ks.launches_by_library)
    ks.linear_swiglu(x.to(DEV), w.to(DEV), silu)
    y = x.double() @ w.double().T
    close(out, plain.gelu_tanh(y[:, :N]) * y[:, N:], 3e-6 if dtype == torch.float32 else 8e-3, "gelu gates")
    close(silu, plain.silu(y[:, :N]) * y[:, N:], 3e-6 if dtype == torch.float32 else 8e-3, "silu gates")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,d,E,top", [(1, 64, 6, 2), (33, 72, 11, 3), (300, 130, 5, 5), (9, 40, 1, 1)])
def test_router_with_a_bias_on_its_logits(dtype, M, d, E, top):
    ks = kernels(dtype)
    g = gen(M + E)
    x, w, b = torch.randn((M, d), generator=g).to(dtype), torch.randn((E, d), generator=g) / d ** 0.5, torch.randn(E, generator=g) * 2.0
    r = ks.moe_route(x.to(DEV), w.to(DEV), top, want_logits=True, scoring="softmax_renorm", logit_bias=b.to(DEV))
    z = x.double() @ w.double().T + b.double()
    close(r.logits, z, 1e-5, "logits")
    order = torch.argsort(r.logits.double().cpu(), dim=-1, descending=True, stable=True)[:, :top]
    assert torch.equal(r.expert_ids.cpu().T.long(), order)
    share = torch.softmax(torch.gather(z, 1, order), -1)
    close(r.weights.T, share, 1e-5, "weights")
    for s in range(top):
        assert torch.equal(r.sorted_weights[s].cpu(), r.weights[s].cpu()[r.sorted_rows[s].cpu().long()])


@pytest.mark.parametrize("M,d", [(1, 72), (5, 33), (300, 1024)])
def test_what_is_added_between_two_passes(M, d):
    from spite_b200.config import PartSpec
    from spite_b200.parts import BuildContext, build_part
    ks, g = kernels(torch.float32), gen(d)
    j = build_part("junction", PartSpec("reinject_add", {"hidden_size": d, "steps": 3}), BuildContext(ks, torch.float32, torch.device(DEV)))
    step, h, h0 = (torch.randn(s, generator=g) for s in ((3, d), (M, d), (M, d)))
    j.bind({"step": step.to(DEV)})
    for t in range(3):
        got = h.to(DEV)
        j.forward(got, h0.to(DEV), None, t)
        assert torch.equal(got.cpu(), (h + h0 if t else h) + step[t])


# ---------------------------------------------------------------------------- the engine
@pytest.fixture(scope="module", params=list(S.CONFIGS))
def folder(request, tmp_path_factory):
    return S.write_model(tmp_path_factory.mktemp(f"fozutar_{request.param}"), request.param), request.param


@pytest.fixture(scope="module", params=["float32", "bfloat16"])
def setup(request, folder, tmp_path_factory):
    from spite_b200.engine import Model
    path, name = folder
    dtype = request.param
    if dtype == "bfloat16":                                  # no choice of experts left to rounding
        path = S.write_model(tmp_path_factory.mktemp(f"fozutar_settled_{name}"), name, settled_routing=True)
    model = Model.from_folder(path, dtype=dtype, device=DEV)
    vocab = model.plan.vocab_size
    lengths = {"a": 210 if name == "G" else 97, "b": 40, "c": 37, "d": 66, "e": 1, "f": 21}
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


def test_the_residual_stream_layer_run_by_layer_run(setup):
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
    the other, every chunk of the configuration crossed while decoding)."""
    path, model, requests, tol, dtype = setup
    reqs = {"long": H.random_tokens(model.plan.vocab_size, 163, 77)}
    steps = H.steps_last_decoded(reqs, 160)
    eng = _engine(model, steps, 16)
    S.compare_with_plain(H.run_steps(eng, steps), path, reqs, tol)
    assert eng.graph_replays > 100


def test_decode_steps_of_many_requests_from_graphs(setup):
    """Eleven requests decode side by side and end one by one: the captured steps' padding rows (copies of the first row, slot
    included) leave states and caches as they were."""
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


def test_trace_replay_program(folder, tmp_path):
    """`bin/trace_run` as a program: a mixed schedule in, logits files out, equal to the plain implementation."""
    import subprocess, sys
    import numpy as np
    from pathlib import Path
    path, name = folder
    if name not in ("F", "G"):
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


def test_the_command_line_runs_a_fozutar_folder(tmp_path):
    """`spite random`, `spite run` (greedy, float32: the plain implementation's tokens) and `spite bench`."""
    import subprocess, sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    spite = lambda *a: subprocess.run([sys.executable, str(root / "bin" / "spite")] + [str(x) for x in a],
                                      capture_output=True, text=True, timeout=900)
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(S.CONFIG_F))
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
