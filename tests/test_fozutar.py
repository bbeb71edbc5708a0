"""Fozutar without a GPU: the configuration and its errors, tensor names and the sizes that only tensors give, the plain
implementation's mechanisms against loops written out element by element, and the engine (cache, state slots, batches, trace
replay) with the plain torch kernel set in every cut."""
import json
import math

import pytest
import torch

import fozutar_helpers as S
import helpers as H
import plain_fozutar as plain
from reference_kernels import TorchReferenceKernels
from spite_b200.cache import Window
from spite_b200.config import ConfigError, FozutarConfig, JunctionCall, load_config
from spite_b200.engine import Engine, Model
from spite_b200.kernels.api import DistanceBias
from spite_b200.parts.position import distance_rows
from spite_b200.weights import WeightError, save_file


# ---------------------------------------------------------------------------- configuration
def test_configuration_round_trip_and_run_order():
    for name, (cfg, _, _) in S.CONFIGS.items():
        c = FozutarConfig.from_dict(cfg)
        assert c.to_dict() == cfg, name
        plan = c.plan()
        assert [b.arrangement for b in plan.blocks] == ["parallel_residual"] * len(cfg["layers"])
        assert plan.tie_word_embeddings and plan.embedding_scale == cfg["embedding"]["scale"]
        assert plan.position_table == plan.max_positions == cfg["max_positions"]
    # three passes over layers 1..3, each begun by the junction, each run with a cache of its own
    plan = FozutarConfig.from_dict(S.CONFIG_F).plan()
    got = [("pass", c.step) if isinstance(c, JunctionCall) else (c.layer, c.cache) for c in plan.order]
    assert got == [(0, 0), ("pass", 0), (1, 1), (2, 2), (3, 3), ("pass", 1), (1, 4), (2, 5), (3, 6), ("pass", 2), (1, 7), (2, 8), (3, 9),
                   (4, 10)]
    assert FozutarConfig.from_dict(S.CONFIG_J).plan().junctions == ()


def test_tensor_names_and_shapes():
    c = FozutarConfig.from_dict(S.CONFIG_F)
    shape = {n: b.source_shape for b in c.weight_bindings() for n in b.sources}
    assert shape["pos"] == (400, 72) and shape["loop.step"] == (3, 72) and shape["embed"] == (211, 72)
    assert shape["l0.mix.a1"] == (5, 72) and shape["l0.mix.a2"] == (30, 5) and shape["l0.mix.norm"] == (14,)
    assert shape["l1.mix.q.b"] == (96,) and shape["l1.mix.k"] == (48, 72) and shape["l1.mix.rel"] == (8, 4)
    assert shape["l1.mlp.router.b"] == (5,) and shape["l1.mlp.e4.down"] == (72, 24) and shape["l0.mlp.gate"] == (40, 72)
    assert not any(n.startswith("l2.mlp") for n in shape) and "l1.mix.v" not in shape and "head" not in shape
    assert "loop.step" not in {n for b in FozutarConfig.from_dict(S.CONFIG_J).weight_bindings() for n in b.sources}


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][1]["mixer"].update(vdim=16), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("softcap"), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][1]["mixer"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][1]["mixer"].update(bias_max=0), "bias_max"),
    (lambda c: c["layers"][0]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0), "tau"),
    (lambda c: c["layers"][0].update(type="delta"), "not a mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="shared"), "mlp.kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
])
def test_configuration_errors_name_the_key(change, word):
    cfg = json.loads(json.dumps(S.CONFIG_F))
    change(cfg)
    with pytest.raises(ConfigError, match=word):
        FozutarConfig.from_dict(cfg)


def test_sizes_that_only_tensors_give(tmp_path):
    """A file without `rank` and `buckets`: both come from the tensors, layer by layer; one that disagrees with itself is
    refused by name."""
    folder = S.write_model(tmp_path, "F")
    cfg = json.loads((folder / "config.json").read_text())
    for L in cfg["layers"]:
        L["mixer"].pop("rank", None)
        L["mixer"].pop("buckets", None)
    (folder / "config.json").write_text(json.dumps(cfg))
    c = load_config(folder)
    assert [getattr(L.mixer, "decay_rank", None) or L.mixer.table_rows for L in c.layers] == [5, 8, 20, 12, 6]
    k = TorchReferenceKernels(torch.float32, "cpu")
    Model.from_folder(folder, dtype="float32", device="cpu", kernels=k)
    _, tensors = plain.load_folder(folder)
    tensors["l0.mix.a2"] = tensors["l0.mix.a2"][:, :4].contiguous()
    save_file(tensors, folder / "model.safetensors")
    with pytest.raises(WeightError, match="l0.mix.a2"):
        Model.from_folder(folder, dtype="float32", device="cpu", kernels=k)


# ---------------------------------------------------------------------------- mechanisms
def test_buckets_of_distances():
    assert [plain.bucket(n, 8, 64) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    for rows, far in ((8, 64), (32, 128), (32, 100), (12, 60), (6, 31), (2, 2), (4, 3), (5, 9), (64, 4096)):
        got = distance_rows(rows, far, 2 * far)
        assert got == [plain.bucket(n, rows, far) for n in range(2 * far)]
        assert got == sorted(got) and got[0] == 0 and got[far] == rows - 1 and got[-1] == rows - 1
    # a far distance within the first half: nothing there changes, and a chunk may end before the second half begins
    assert distance_rows(8, 4, 6) == [0, 1, 2, 3, 7, 7] and distance_rows(8, 3, 4) == [0, 1, 2, 3] and distance_rows(1, 5, 3) == [0, 0, 0]
    for rows, far in ((0, 5), (8, 0)):
        with pytest.raises(ConfigError):
            distance_rows(rows, far, 10)


def test_numbers_by_distance_are_laid_out_with_repeated_ends():
    table = torch.randn(6, 3)
    rows = distance_rows(6, 31, 32)
    d = DistanceBias.from_rows(table, rows)
    P = d.PAD
    assert d.length == 32 and d.padded.shape == (3, 32 + 2 * P)
    for n in range(-P, 32 + P):
        assert torch.equal(d.padded[:, P + n], table[rows[min(max(n, 0), 31)]])
    runs = d.runs.tolist()
    for n in range(32):
        assert rows[runs[n]] == rows[n] and (runs[n] == 0 or rows[runs[n] - 1] != rows[n])


def test_attention_of_the_plain_implementation_element_by_element():
    mx = {"heads": 4, "kv_heads": 2, "dim": 6, "scale": 0.7, "softcap": 1.5, "bias_max": 9, "mask": {"size": 5}}
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(s, generator=g, dtype=torch.float64)
    w = {"q": r(24, 10), "q.b": r(24), "k": r(12, 10), "k.b": r(12), "rel": r(4, 4), "o": torch.eye(24, dtype=torch.float64)}
    h, eps, T = r(13, 10), 1e-3, 13
    out = plain.attention(h, w, mx, eps).view(T, 4, 6)
    norm = lambda u: u / math.sqrt(float((u * u).mean()) + eps)
    for i in (0, 4, 5, 9, 12):
        for hd in range(4):
            kv = hd // 2
            qi = norm(w["q"][hd * 6:hd * 6 + 6] @ h[i] + w["q.b"][hd * 6:hd * 6 + 6])
            num, den = torch.zeros(6, dtype=torch.float64), 0.0
            for j in range(i // 5 * 5, i + 1):
                kj = w["k"][kv * 6:kv * 6 + 6] @ h[j] + w["k.b"][kv * 6:kv * 6 + 6]
                s = 1.5 * math.tanh(0.7 * float(qi @ norm(kj)) / 1.5) + float(w["rel"][plain.bucket(i - j, 4, 9), hd])
                num, den = num + math.exp(s) * kj, den + math.exp(s)
            assert torch.allclose(out[i, hd], num / den, atol=1e-12)


def test_gated_linear_attention_against_its_closed_form():
    """o_t = sum over s <= t of (q_t . (prod of the decays after s) k_s) v_s, the token itself undecayed."""
    mx, eps, T = {"heads": 2, "dim": 3, "vdim": 4, "tau": 5.0}, 1e-4, 7
    g = torch.Generator().manual_seed(2)
    r = lambda *s: torch.randn(s, generator=g, dtype=torch.float64)
    w = {"q": r(6, 5), "k": r(6, 5), "v": r(8, 5), "g": r(8, 5), "a1": r(2, 5), "a2": r(6, 2), "a2.b": r(6), "norm": r(4),
         "o": torch.eye(8, dtype=torch.float64)}
    h = r(T, 5)
    out = plain.gla(h, w, mx, eps)
    alpha = torch.sigmoid(h @ w["a1"].T @ w["a2"].T + w["a2.b"]) ** 0.2
    for t in range(T):
        for hd in range(2):
            K, V = slice(hd * 3, hd * 3 + 3), slice(hd * 4, hd * 4 + 4)
            o = torch.zeros(4, dtype=torch.float64)
            for s in range(t + 1):
                d = torch.ones(3, dtype=torch.float64)
                for u in range(s + 1, t + 1):
                    d = d * alpha[u, K]
                o = o + float((w["q"][K] @ h[t] / math.sqrt(3.0) * d * (w["k"][K] @ h[s])).sum()) * (w["v"][V] @ h[s])
            o = o / math.sqrt(float((o * o).mean()) + eps) * w["norm"]
            z = w["g"][V] @ h[t]
            assert torch.allclose(out[t, V], o * z / (1 + torch.exp(-z)), atol=1e-10)


def test_router_takes_the_largest_biased_logits():
    ff = {"router": {"experts": 3, "top": 2}}
    w = {"router": torch.zeros(3, 4, dtype=torch.float64), "router.b": torch.tensor([0.0, 0.0, 1.5], dtype=torch.float64)}
    w["router"][0, 0], w["router"][1, 0] = 2.0, 1.0
    g = torch.Generator().manual_seed(3)
    for e in range(3):
        for n, s in (("gate", (5, 4)), ("up", (5, 4)), ("down", (4, 5))):
            w[f"e{e}.{n}"] = torch.randn(s, generator=g, dtype=torch.float64)
    h = torch.tensor([[1.0, 0.5, -0.3, 0.2]], dtype=torch.float64)
    expert = lambda e: (plain.silu(h[0] @ w[f"e{e}.gate"].T) * (h[0] @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T
    p = 1.0 / (1.0 + math.exp(-0.5))                                      # the softmax over the chosen logits 2.0 and 1.5
    assert torch.allclose(plain.moe(h, w, ff)[0], p * expert(0) + (1 - p) * expert(2))


# ---------------------------------------------------------------------------- the engine on the host
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {n: S.write_model(tmp_path_factory.mktemp(f"fozutar_{n}"), n) for n in ("F", "H")}


def host_engine(folder, tokens, page_size=16, max_requests=4):
    k = TorchReferenceKernels(torch.float32, "cpu")
    model = Model.from_folder(folder, dtype="float32", device="cpu", kernels=k)
    return Engine(model, cache_tokens=tokens, page_size=page_size, max_requests=max_requests)


def requests_for(folder, lens, seed):
    vocab = json.loads((folder / "config.json").read_text())["vocab"]
    return {f"r{i}": H.random_tokens(vocab, n, seed + i) for i, n in enumerate(lens)}


@pytest.mark.parametrize("name", ["F", "H"])
def test_whole_prompts_and_the_stream_after_every_layer_run(folders, name):
    folder = folders[name]
    assert load_config(folder).to_dict() == S.CONFIGS[name][0]
    reqs = requests_for(folder, (47, 1, 20), 10)
    eng = host_engine(folder, 64 * 3)
    S.compare_with_plain(H.run_steps(eng, H.steps_whole(reqs)), folder, reqs, 2e-5)
    assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups
    cfg, tensors = S.folder_contents(str(folder))
    taps, seen = [], []
    plain.forward(cfg, tensors, reqs["r0"], taps=taps)
    eng.model.layer_tap = lambda i, h: seen.append(h.clone())
    H.run_steps(eng, H.steps_whole({"r0": reqs["r0"]}))
    assert len(seen) == len(taps) == len(plain.runs(cfg))
    for i, h in enumerate(seen):
        assert float((h - taps[i]).abs().max()) <= 3e-5 * float(taps[i].abs().max()), f"layer run {i}"


@pytest.mark.parametrize("name", ["F", "H"])
def test_portions_decoding_and_mixed_batches_on_the_host(folders, name):
    """Token by token after a prompt, portions down to two tokens, and up to four live requests in a pool that forces pages
    and state slots to be used again: the logits are those of the whole sequence."""
    folder = folders[name]
    reqs = requests_for(folder, (45, 9, 30, 3, 26), 30)
    cuts = {"decoded": H.steps_last_decoded(reqs, 12), "portions": H.steps_portions(reqs, seed=2),
            "mixed": H.steps_mixed(reqs, {r: max(1, len(t) - 6) for r, t in reqs.items()}, seed=3)}
    for what, steps in cuts.items():
        eng = host_engine(folder, H.max_tokens_of(steps) if what == "mixed" else 64, page_size=16)
        S.compare_with_plain(H.run_steps(eng, steps), folder, reqs, 2e-5)
        assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups, what


def test_caches_and_state_of_every_layer_run(folders):
    """Chunks of two sizes get page groups of their own, every pass through the loop keys and matrices of its own."""
    k = TorchReferenceKernels(torch.float32, "cpu")
    model = Model.from_config(FozutarConfig.from_dict(S.CONFIG_F), dtype="float32", device="cpu", kernels=k)
    specs = model.cache_specs()
    assert sorted(specs) == list(range(11))
    for run in (1, 4, 7):
        assert specs[run][0].window == Window("chunk", 20) and specs[run][1] is None
        assert specs[run][0].planes == 1 and specs[run][0].key_scales       # one row a position, and its factor
        assert specs[run + 1] [0] is None and specs[run + 1][1].shape == (2 * 7 * 36,)
        assert specs[run + 2][0].window == Window("chunk", 33)
    assert specs[0][1].shape == (3 * 14 * 12,) and specs[10][0].window == Window("chunk", 50)


def test_pages_behind_a_chunk_go_back_and_a_used_slot_starts_at_zero(folders):
    eng = host_engine(folders["F"], 256, page_size=8, max_requests=1)
    toks = requests_for(folders["F"], (90,), 50)["r0"]
    H.run_steps(eng, [{"step": 0, "entries": [{"id": "a", "tokens": toks, "want": [89]}], "end": []}])
    by_window = {k.window: g for g, k in enumerate(eng.storage.group_keys)}
    for size, first in ((20, 80), (33, 66), (50, 50)):
        held = [p >= 0 for p in eng.cache.block_table("a", by_window[Window("chunk", size)])]
        assert held == [8 * i + 7 >= first for i in range(12)], size
    eng.finish("a")
    reqs = requests_for(folders["F"], (30, 25), 60)
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": reqs["r0"], "want": [29]}], "end": ["r0"]},
             {"step": 1, "entries": [{"id": "r1", "tokens": reqs["r1"][:10], "want": [9]}], "end": []},
             {"step": 2, "entries": [{"id": "r1", "tokens": reqs["r1"][10:], "want": [0, 14]}], "end": ["r1"]}]
    S.compare_with_plain(H.run_steps(eng, steps), folders["F"], reqs, 2e-5)


def test_positions_end_with_the_table(folders):
    from spite_b200.engine import ContextOverflow
    eng = host_engine(folders["H"], 256)
    toks = requests_for(folders["H"], (181,), 5)["r0"]
    with pytest.raises(ContextOverflow):
        H.run_steps(eng, H.steps_whole({"a": toks}))


def test_trace_replay_on_the_host(folders, tmp_path):
    import io
    import numpy as np
    from spite_b200.engine.trace import replay
    folder = folders["F"]
    reqs = requests_for(folder, (50, 21, 5), 70)
    steps = H.steps_mixed(reqs, {r: len(t) - 4 for r, t in reqs.items()}, seed=9)
    eng = host_engine(folder, H.max_tokens_of(steps), page_size=64)
    log = io.StringIO()
    replay(eng, [json.dumps(s) for s in steps], tmp_path / "out", log=log)
    assert log.getvalue().split("\n")[:-1] == [f"done {s['step']}" for s in steps]
    vocab = S.CONFIG_F["vocab"]
    pos, got = {}, {}
    for s in steps:
        if not any(e["want"] for e in s["entries"]):
            continue
        rows = np.fromfile(tmp_path / "out" / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab)
        i = 0
        for e in s["entries"]:
            base = pos.get(e["id"], 0)
            for w in e["want"]:
                got[(e["id"], base + w)] = torch.from_numpy(rows[i].copy())
                i += 1
            pos[e["id"]] = base + len(e["tokens"])
    S.compare_with_plain(got, folder, reqs, 2e-5)
