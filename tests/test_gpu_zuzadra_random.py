"""Random Zuzadra configurations on the GPU: width, vocabulary, number of streams, layer order, a looped range or none, head
counts and sizes (no multiples of 16, value heads larger and smaller than key heads, more query heads per kv head than the
tensor-core kernels take), rotations of two elements up to the whole head, windows shorter than a page, longer than the prompts
or none, state spaces of 1 to 200 key rows in several groups and norm parts with one to eight taps, decays of any inner size,
scales of either sign and missing feed-forwards are drawn per seed; then the engine runs whole prompts, portions, decoding and
a mixed schedule in float32 (bit-identical between the cuts) and in bfloat16 against the plain implementation."""
import random

import pytest
import torch

import helpers as H
import zuzadra_helpers as S
from zuzadra_helpers import _layer, _left, _model, _par, _ssm

pytestmark = pytest.mark.gpu

DEV = "cuda:0"


def random_config(seed: int) -> dict:
    rng = random.Random(7000 + seed)
    width = rng.choice([40, 64, 72, 100, 128, 200, 256, 320])
    layers = []
    for i in range(rng.randint(2, 6)):
        ff = rng.choice([None, 8, 24, 40, 64, 100, 128])
        if rng.random() < 0.5:
            heads = rng.choice([1, 2, 3, 4, 6, 8])
            vdim = rng.choice([4, 5, 8, 12, 16, 32, 48, 64, 70])
            parts = rng.choice([p for p in (1, 2, 3, 4, heads) if (heads * vdim) % p == 0])
            groups = rng.choice([g for g in range(1, heads + 1) if heads % g == 0])
            mixer = _ssm(heads, vdim, rng.choice([1, 4, 10, 16, 32, 33, 48, 64, 100, 128, 200]), groups, rng.choice([1, 2, 3, 4, 4, 8]), parts)
        else:
            heads = rng.choice([1, 2, 3, 4, 6, 8, 20])
            kv = rng.choice([k for k in range(1, heads + 1) if heads % k == 0])
            dim, vdim = rng.choice([8, 10, 16, 24, 32, 40, 48, 64, 80, 128]), rng.choice([2, 8, 10, 16, 24, 32, 48, 64, 96, 128])
            dims = rng.choice([d for d in (2, 4, 6, 8, 10, 16, 24, 32, 64, 128, dim) if d <= dim])
            left = _left(heads, kv, dim, vdim, round(rng.uniform(0.5, 1.5) / dim ** 0.5, 4), dims, rng.choice([10.0, 1e4, 5e5]),
                         rng.choice([None, 1, 5, 16, 33, 40, 64, 100, 128, 200, 1000]))
            mixer = _par(left, rng.choice([1, 2, 3, 5]), rng.choice([4, 6, 16, 32, 33, 48, 64, 100]), rng.choice([1, 3, 8, 20, 64]),
                         rng.choice([0.5, 1.0, 1.3, -0.8]), rng.choice([0.4, 1.0, 1.2, -1.1]))
        layers.append(_layer(mixer, ff))
    loop = None
    if rng.random() < 0.6:
        start = rng.randrange(len(layers))
        stop = rng.randint(start + 1, len(layers))
        loop = (start, stop, rng.choice([1, 2, 2, 3]) if stop - start < 4 else 2)
    return _model(rng.choice([101, 256, 517, 1000]), width, rng.choice([1e-6, 1e-5, 1e-3]), rng.choice([1, 2, 3, 3, 4, 6]), layers, loop)


N_CONFIGS = 10


@pytest.fixture(scope="module", params=range(N_CONFIGS))
def model_folder(request, tmp_path_factory):
    seed = request.param
    cfg = random_config(seed)
    S.CONFIGS[f"random{seed}"] = (cfg, 0.08, seed)
    try:
        folder = S.write_model(tmp_path_factory.mktemp(f"zuzadra_random_{seed}"), f"random{seed}")
    finally:
        del S.CONFIGS[f"random{seed}"]
    return folder, cfg, seed


def _run(model, steps, page):
    from spite_b200.engine import Engine
    eng = Engine(model, cache_tokens=H.max_tokens_of(steps), page_size=page, max_requests=4)
    out = H.run_steps(eng, steps)
    eng.check()
    assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups
    return out


def test_float32_every_cut(model_folder):
    from spite_b200.engine import Model
    folder, cfg, seed = model_folder
    model = Model.from_folder(folder, dtype="float32", device=DEV)
    reqs = {r: H.random_tokens(cfg["vocab"], n, seed * 10 + i) for i, (r, n) in enumerate({"a": 180, "b": 33, "c": 1, "d": 58}.items())}
    n_prompt = {r: max(1, len(t) - 7) for r, t in reqs.items()}
    cuts = {"whole": _run(model, H.steps_whole(reqs), 64), "portions": _run(model, H.steps_portions(reqs, seed=seed), 16),
            "decoded": _run(model, H.steps_last_decoded(reqs, 40), 64),
            "mixed": _run(model, H.steps_mixed(reqs, n_prompt, seed=seed), 16)}
    for res in cuts.values():
        S.compare_with_plain(res, folder, reqs, 4e-5)
    H.assert_cuts_identical(cuts)


def test_bfloat16_every_cut(model_folder):
    from spite_b200.engine import Model
    folder, cfg, seed = model_folder
    model = Model.from_folder(folder, dtype="bfloat16", device=DEV)
    reqs = {r: H.random_tokens(cfg["vocab"], n, seed * 10 + i) for i, (r, n) in enumerate({"a": 130, "b": 33, "c": 1}.items())}
    n_prompt = {r: max(1, len(t) - 7) for r, t in reqs.items()}
    for steps, page in ((H.steps_whole(reqs), 64), (H.steps_portions(reqs, seed=seed), 16), (H.steps_last_decoded(reqs, 40), 64),
                        (H.steps_mixed(reqs, n_prompt, seed=seed), 64)):
        res = _run(model, steps, page)
        S.compare_with_plain(res, folder, reqs, 3e-2)
        ref, rounding = S.plain_logits(folder, reqs["a"], sixteen=True)
        errs = torch.tensor([float((res[("a", p)].double().cpu() - ref[p]).abs().max()) for p in range(len(reqs["a"]))]) / float(ref.abs().max())
        allowed = max(2e-2, float(rounding.median()))
        assert float(errs.median()) <= allowed, f"median error {float(errs.median()):.3e} exceeds {allowed:.1e}"
