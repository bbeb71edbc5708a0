"""Random Fozutar configurations on the GPU: width, vocabulary, layer order, a looped range or none, head counts and sizes (odd
ones, no multiples of 16, more query heads per kv head than the tensor-core kernels take), chunks from one position to more than
the prompts, tables by distance of two to forty rows that end inside the chunk or beyond it, memories of 1 to 200 key rows with
decays of any inner size and root, one to nine experts, dense feed-forwards and none are drawn per seed; then the engine runs
whole prompts, portions, decoding and a mixed schedule in float32 (bit-identical between the cuts) and in bfloat16 against the
plain implementation."""
import random

import pytest
import torch

import fozutar_helpers as S
import helpers as H
from fozutar_helpers import _attn, _dense, _gla, _layer, _model, _moe

pytestmark = pytest.mark.gpu

DEV = "cuda:0"


def random_config(seed: int) -> dict:
    rng = random.Random(8000 + seed)
    width = rng.choice([40, 64, 72, 100, 128, 200, 256, 320])
    layers = []
    for i in range(rng.randint(2, 5)):
        if rng.random() < 0.5:
            mixer = _gla(rng.choice([1, 2, 3, 4, 6]), rng.choice([2, 4, 10, 16, 32, 33, 48, 64, 100, 128, 200]),
                         rng.choice([4, 5, 8, 12, 16, 32, 48, 64, 70]), rng.choice([1.0, 2.5, 8.0, 16.0, 40.0]), rng.choice([1, 3, 8, 16, 20, 64, 70]))
        else:
            heads = rng.choice([1, 2, 3, 4, 6, 8, 20])
            kv = rng.choice([k for k in range(1, heads + 1) if heads % k == 0])
            dim = rng.choice([7, 8, 10, 16, 24, 32, 40, 48, 64, 64, 80, 128, 128])
            chunk = rng.choice([1, 5, 16, 33, 40, 64, 100, 128, 200, 1000])
            rows = rng.choice([2, 4, 7, 8, 16, 32, 40])
            far = rng.choice([f for f in (3, 9, 17, 25, 60, 100, 128, 256, 1000, chunk) if f > rows // 2])
            mixer = _attn(heads, kv, dim, round(rng.uniform(0.5, 2.0) / dim ** 0.5, 4), rng.choice([1.0, 3.0, 10.0, 50.0]), chunk, far, rows)
        experts = rng.choice([1, 2, 3, 4, 6, 9])
        mlp = rng.choice([None, _dense(rng.choice([8, 24, 40, 100, 128])),
                          _moe(rng.choice([8, 24, 40, 64]), experts, rng.randint(1, min(4, experts)))])
        layers.append(_layer(mixer, mlp))
    loop = None
    if rng.random() < 0.7:
        start = rng.randrange(len(layers))
        stop = rng.randint(start + 1, len(layers))
        loop = (start, stop, rng.choice([1, 2, 2, 3]) if stop - start < 4 else 2)
    return _model(rng.choice([101, 256, 517, 1000]), width, rng.choice([1e-6, 1e-5, 1e-3]), rng.choice([0.5, 1.0, 3.0, 9.0]), rng.choice([180, 256, 777]),
                  layers, loop)


N_CONFIGS = 10


@pytest.fixture(scope="module", params=range(N_CONFIGS))
def model_folders(request, tmp_path_factory):
    seed = request.param
    cfg = random_config(seed)
    S.CONFIGS[f"random{seed}"] = (cfg, 0.08, seed)
    try:
        folders = [S.write_model(tmp_path_factory.mktemp(f"fozutar_random_{seed}"), f"random{seed}", settled_routing=settled)
                   for settled in (False, True)]
    finally:
        del S.CONFIGS[f"random{seed}"]
    return folders, cfg, seed


def _run(model, steps, page):
    from spite_b200.engine import Engine
    eng = Engine(model, cache_tokens=H.max_tokens_of(steps), page_size=page, max_requests=4)
    out = H.run_steps(eng, steps)
    eng.check()
    assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups
    return out


def test_float32_every_cut(model_folders):
    from spite_b200.engine import Model
    (folder, _), cfg, seed = model_folders
    model = Model.from_folder(folder, dtype="float32", device=DEV)
    reqs = {r: H.random_tokens(cfg["vocab"], n, seed * 10 + i) for i, (r, n) in enumerate({"a": 150, "b": 33, "c": 1, "d": 58}.items())}
    n_prompt = {r: max(1, len(t) - 7) for r, t in reqs.items()}
    cuts = {"whole": _run(model, H.steps_whole(reqs), 64), "portions": _run(model, H.steps_portions(reqs, seed=seed), 16),
            "decoded": _run(model, H.steps_last_decoded(reqs, 40), 64),
            "mixed": _run(model, H.steps_mixed(reqs, n_prompt, seed=seed), 16)}
    for res in cuts.values():
        S.compare_with_plain(res, folder, reqs, 4e-5)
    H.assert_cuts_identical(cuts)


def test_bfloat16_every_cut(model_folders):
    from spite_b200.engine import Model
    (_, folder), cfg, seed = model_folders
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
