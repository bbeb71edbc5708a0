"""Zuzadra without a GPU: the configuration and its errors, the size that only a tensor gives, tensor names, the plain
implementation's mechanisms against sums written out element by element, and the engine (cache, state slots, batches, trace
replay) with the plain torch kernel set in every cut."""
import io
import json
import math

import numpy as np
import pytest
import torch

import helpers as H
import plain_zuzadra as plain
import zuzadra_helpers as S
from reference_kernels import TorchReferenceKernels
from spite_b200.cache import Window
from spite_b200.config import ConfigError, PartSpec, ZuzadraConfig, load_config
from spite_b200.engine import Engine, Model
from spite_b200.parts import BuildContext, build_part
from spite_b200.weights import WeightError


# ---------------------------------------------------------------------------- configuration
def test_configuration_round_trip_and_plan():
    for name, (cfg, _, _) in S.CONFIGS.items():
        c = ZuzadraConfig.from_dict(cfg)
        assert c.to_dict() == cfg, name
        plan = c.plan()
        assert {b.arrangement for b in plan.blocks} == {"hyper_residual"} and len(plan.blocks) == len(cfg["layers"])
        assert plan.streams == cfg["streams"] and not plan.tie_word_embeddings
    order = ZuzadraConfig.from_dict(S.CONFIG_P).plan().order
    assert [c.layer for c in order] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [c.cache for c in order] == list(range(11))            # every pass of a looped layer has a cache of its own
    assert [c.layer for c in ZuzadraConfig.from_dict(S.CONFIG_S).plan().order] == [0, 1]


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=15), "vdim"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][2].update(type="mamba"), "not a mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "mlp.kind"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c["norm"].update(eps=0), "eps"),
])
def test_configuration_errors_name_the_key(change, word):
    cfg = json.loads(json.dumps(S.CONFIG_P))
    change(cfg)
    with pytest.raises(ConfigError, match=word):
        ZuzadraConfig.from_dict(cfg)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {n: S.write_model(tmp_path_factory.mktemp(f"zuzadra_{n}"), n) for n in ("P", "R", "S")}


def host_engine(folder, tokens, page_size=16, max_requests=4):
    k = TorchReferenceKernels(torch.float32, "cpu")
    model = Model.from_folder(folder, dtype="float32", device="cpu", kernels=k)
    return Engine(model, cache_tokens=tokens, page_size=page_size, max_requests=max_requests)


def requests_for(folder, lens, seed):
    vocab = json.loads((folder / "config.json").read_text())["vocab"]
    return {f"r{i}": H.random_tokens(vocab, n, seed + i) for i, n in enumerate(lens)}


def test_a_size_that_only_the_tensor_gives(folders, tmp_path):
    """The decay's inner size stands in no config.json: the folder's tensor decides, whatever a default would say; tensors
    of a second sublayer that the layer lacks are passed over; a tensor of another shape is named."""
    raw = json.loads((folders["P"] / "config.json").read_text())
    for L in raw["layers"]:
        if L["type"] == "parallel":
            del L["mixer"]["right"]["rank"]
    assert ZuzadraConfig.from_dict(raw).layers[1].mixer.right.decay_rank == 32
    bare = tmp_path / "bare"
    bare.mkdir()
    (bare / "config.json").write_text(json.dumps(raw))
    tensors = S.folder_contents(str(folders["P"]))[1]
    from spite_b200.weights import save_file
    extra = dict(tensors, **{"l2.norm2": torch.zeros(72, dtype=torch.bfloat16), "l2.hc2.mix": torch.zeros((2, 2), dtype=torch.bfloat16)})
    save_file(extra, bare / "model.safetensors")
    cfg = load_config(bare)
    assert [L.mixer.right.decay_rank for L in cfg.layers if L.type == "parallel"] == [5, 12]
    assert cfg.to_dict() == raw
    toks = H.random_tokens(211, 20, 4)
    S.compare_with_plain(H.run_steps(host_engine(bare, 64), H.steps_whole({"a": toks})), folders["P"], {"a": toks}, 2e-5)
    k = TorchReferenceKernels(torch.float32, "cpu")
    model = Model.from_tensors(ZuzadraConfig.from_dict(raw), tensors, dtype="float32", device="cpu", kernels=k)
    assert model.blocks[1].mixer.sides["right"].rank == 5
    save_file(dict(tensors, **{"l1.mix.right.w2": torch.zeros((30, 6), dtype=torch.bfloat16)}), bare / "model.safetensors")
    with pytest.raises(WeightError, match="l1.mix.right.w2"):
        host_engine(bare, 64)


def test_two_mixers_that_want_the_same_kind_of_cache_are_refused():
    k = TorchReferenceKernels(torch.float32, "cpu")
    ctx = BuildContext(kernels=k, dtype=torch.float32, device=torch.device("cpu"))
    memory = PartSpec("decay_memory", {"hidden_size": 16, "num_heads": 2, "head_dim": 4, "decay_rank": 4, "norm_eps": 1e-5})
    with pytest.raises(ConfigError, match="same kind of cache"):
        build_part("mixer", PartSpec("parallel_mixers", {"hidden_size": 16, "left": memory, "right": memory}), ctx)


def test_what_the_layers_keep(folders):
    eng = host_engine(folders["P"], 64)
    specs = eng.model.cache_specs()
    kv, state = specs[1]                                           # the parallel layer: pages and a slot
    assert kv.window == Window("sliding", 20) and (kv.num_kv_heads, kv.head_dim) == (2, 24)
    assert state.shape == (3 * 10 * 12 + 72,)                      # three matrices of 10 columns by 12 padded rows, the last input
    assert specs[3][0].window == Window("full")
    kv, state = specs[0]                                           # a state space: a slot alone
    assert kv is None and state.shape == (6 * 20 * 20 + 2 * (120 + 2 * 3 * 18),)


# ---------------------------------------------------------------------------- the plain implementation's mechanisms
def test_values_enter_turned_by_their_distance():
    """A value turned by its position and the result turned back by the query's: what counts is the distance."""
    torch.manual_seed(0)
    T, size, base = 9, 6, 40.0
    v = torch.randn(T, 1, size).double()
    p = torch.softmax(torch.randn(T, T).double(), -1)
    turned = plain.rotate_halves(v, size, base)[:, 0]
    got = plain.rotate_halves((p @ turned)[:, None], size, base, sign=-1.0)[:, 0]
    for i in range(T):
        want = torch.zeros(size).double()
        for j in range(T):
            for m in range(size // 2):
                a = (j - i) * base ** (-2.0 * m / size)
                x, y = float(v[j, 0, m]), float(v[j, 0, m + size // 2])
                want[m] += p[i, j] * (x * math.cos(a) - y * math.sin(a))
                want[m + size // 2] += p[i, j] * (y * math.cos(a) + x * math.sin(a))
        assert float((got[i] - want).abs().max()) < 1e-12


def test_window_sees_the_token_and_those_just_before_it():
    see = plain.window_mask(6, 3)
    assert see[0].tolist() == [True] + [False] * 5
    assert see[4].tolist() == [False, False, True, True, True, False]
    assert plain.window_mask(4, 1).tolist() == torch.eye(4, dtype=torch.bool).tolist()


def test_state_space_against_its_closed_form():
    """y_t = sum over s <= t of exp(-exp(A) (dt_(s+1) + .. + dt_t)) dt_s (B_s . C_t) x_s + D x_t."""
    torch.manual_seed(1)
    T, d, H_, P, N, G, taps = 8, 10, 4, 3, 5, 2, 3
    inner, ch = H_ * P, H_ * P + 2 * G * N
    rnd = lambda *s: torch.randn(*s).double()
    w = {"in": rnd(2 * inner + 2 * G * N + H_, d), "conv": rnd(ch, taps), "conv.b": rnd(ch), "dt_bias": rnd(H_), "A_log": rnd(H_),
         "D": rnd(H_), "norm": rnd(inner), "o": rnd(d, inner)}
    h = rnd(T, d)
    mx = {"heads": H_, "vdim": P, "state": N, "groups": G, "norm_groups": 2}
    got = plain.state_space(h, w, mx, 1e-4)
    proj = h @ w["in"].T
    z, raw, dt = proj[:, :inner], proj[:, inner:inner + ch], torch.log1p(torch.exp(proj[:, inner + ch:] + w["dt_bias"]))
    act = torch.zeros(T, ch).double()
    for t in range(T):
        for c in range(ch):
            s = float(w["conv.b"][c]) + sum(float(w["conv"][c, j]) * float(raw[t - taps + 1 + j, c]) for j in range(taps) if t - taps + 1 + j >= 0)
            act[t, c] = s / (1.0 + math.exp(-s))
    out = torch.zeros(T, inner).double()
    for a in range(H_):
        g = a // (H_ // G)
        x = act[:, a * P:(a + 1) * P]
        B, C = act[:, inner + g * N:inner + (g + 1) * N], act[:, inner + (G + g) * N:inner + (G + g + 1) * N]
        for t in range(T):
            y = w["D"][a] * x[t]
            for s in range(t + 1):
                y = y + torch.exp(-torch.exp(w["A_log"][a]) * dt[s + 1:t + 1, a].sum()) * dt[s, a] * (B[s] @ C[t]) * x[s]
            out[t, a * P:(a + 1) * P] = y
    out = out * z / (1.0 + torch.exp(-z))
    half = inner // 2
    for part in (slice(0, half), slice(half, inner)):
        out[:, part] = out[:, part] / torch.sqrt((out[:, part] ** 2).mean(-1, keepdim=True) + 1e-4)
    ref = (out * w["norm"]) @ w["o"].T
    assert float((got - ref).abs().max()) < 1e-10 * float(ref.abs().max())


def test_decaying_memory_against_its_closed_form():
    """o_t = sum over s < t of (sum_i r_i (w_(s+1) .. w_(t-1))_i k_s,i) v_s + (sum_i r_i u_i k_t,i) v_t."""
    torch.manual_seed(2)
    T, d, H_, n, rank = 7, 9, 2, 4, 3
    rnd = lambda *s: torch.randn(*s).double()
    w = {s: rnd(H_ * n, d) for s in "rkvg"}
    w.update({"mu." + s: torch.rand(d).double() for s in "rkvgw"})
    w.update({"w1": rnd(rank, d), "w2": rnd(H_ * n, rank), "w0": rnd(H_ * n), "u": rnd(H_, n), "norm": rnd(H_ * n), "o": rnd(d, H_ * n)})
    h = rnd(T, d)
    got = plain.decay_attention(h, w, {"heads": H_, "dim": n}, 1e-3)
    m = {s: torch.stack([h[t] + ((h[t - 1] if t else torch.zeros(d).double()) - h[t]) * w["mu." + s] for t in range(T)]) for s in "rkvgw"}
    r, k, v, g = (m[s] @ w[s].T for s in "rkvg")
    dec = torch.exp(-torch.exp(torch.tanh(m["w"] @ w["w1"].T) @ w["w2"].T + w["w0"]))
    out = torch.zeros(T, H_ * n).double()
    for a in range(H_):
        c = slice(a * n, (a + 1) * n)
        for t in range(T):
            o = (r[t, c] * w["u"][a] * k[t, c]).sum() * v[t, c]
            for s in range(t):
                o = o + (r[t, c] * dec[s + 1:t, c].prod(0) * k[s, c]).sum() * v[s, c]
            out[t, c] = o / torch.sqrt((o * o).mean() + 1e-3)
    ref = (out * w["norm"] * g / (1.0 + torch.exp(-g))) @ w["o"].T
    assert float((got - ref).abs().max()) < 1e-10 * float(ref.abs().max())


def test_streams_mix_from_the_old_ones_at_once():
    X = [torch.tensor([[1.0, 2.0]]), torch.tensor([[10.0, 20.0]])]
    mix = torch.tensor([[0.5, 2.0], [3.0, -1.0]])                  # [from, to]
    y = torch.tensor([[100.0, 0.0]])
    new = plain.mix_streams(X, y, mix, torch.tensor([1.0, -1.0]))
    assert new[0].tolist() == [[0.5 * 1 + 3 * 10 + 100, 0.5 * 2 + 3 * 20]]
    assert new[1].tolist() == [[2.0 * 1 - 10 - 100, 2.0 * 2 - 20]]


def test_xielu_at_some_points():
    p, q = (torch.tensor(v, dtype=torch.float64) for v in (0.3, -0.7))
    ap, an = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.7))
    for z in (-30.0, -2.0, -1e-3, 0.0, 1e-3, 0.5, 4.0):
        want = ap * z * z + z / 2 if z > 0 else an * (math.exp(z) - 1 - z) + z / 2
        assert abs(float(plain.xielu(torch.tensor(z, dtype=torch.float64), p, q)) - want) < 1e-12


# ---------------------------------------------------------------------------- the engine on the host
@pytest.mark.parametrize("name", ["P", "R", "S"])
def test_folder_round_trip_and_whole_prompts(folders, name):
    folder = folders[name]
    assert load_config(folder).to_dict() == S.CONFIGS[name][0]
    reqs = requests_for(folder, (47, 1, 20), 10)
    eng = host_engine(folder, 64 * 3)
    S.compare_with_plain(H.run_steps(eng, H.steps_whole(reqs)), folder, reqs, 2e-5)
    assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups


def test_the_sum_of_the_streams_after_every_layer_run(folders):
    folder = folders["P"]
    toks = requests_for(folder, (45,), 20)["r0"]
    cfg, tensors = S.folder_contents(str(folder))
    taps = []
    plain.forward(cfg, tensors, toks, taps=taps)
    eng = host_engine(folder, 64)
    seen = []
    eng.model.layer_tap = lambda i, h: seen.append(h.clone())
    H.run_steps(eng, H.steps_whole({"a": toks}))
    assert len(seen) == len(taps) == 11
    for i, h in enumerate(seen):
        assert float((h - taps[i]).abs().max()) <= 2e-5 * float(taps[i].abs().max()), f"layer run {i}"


@pytest.mark.parametrize("name", ["P", "R"])
def test_portions_decoding_and_mixed_batches_on_the_host(folders, name):
    """Token by token after a prompt, portions down to two tokens, and up to four live requests in a pool that
    forces pages and state slots to be used again: the logits are those of the whole sequence."""
    folder = folders[name]
    reqs = requests_for(folder, (45, 9, 3, 26, 17), 30)
    cuts = {"decoded": H.steps_last_decoded(reqs, 12), "portions": H.steps_portions(reqs, seed=2),
            "mixed": H.steps_mixed(reqs, {r: max(1, len(t) - 6) for r, t in reqs.items()}, seed=3)}
    for what, steps in cuts.items():
        eng = host_engine(folder, H.max_tokens_of(steps) if what == "mixed" else 64, page_size=16)
        S.compare_with_plain(H.run_steps(eng, steps), folder, reqs, 2e-5)
        assert eng.cache.free_pages() == [eng.n_pages] * eng.storage.n_groups, what


def test_pages_behind_a_window_go_back_pass_by_pass(folders):
    """The looped range runs three times: three caches with the window of 20 in one group, three that keep every key."""
    eng = host_engine(folders["P"], 256, page_size=8)
    toks = requests_for(folders["P"], (90,), 50)["r0"]
    H.run_steps(eng, [{"step": 0, "entries": [{"id": "a", "tokens": toks, "want": [89]}], "end": []}])
    by_window = {k.window: g for g, k in enumerate(eng.storage.group_keys)}
    table = eng.cache.block_table("a", by_window[Window("sliding", 20)])
    assert [p >= 0 for p in table] == [False] * 8 + [True] * 4            # the next token still reads positions 71 .. 89
    assert all(p >= 0 for p in eng.cache.block_table("a", by_window[Window("full")]))
    assert eng.storage.kv[by_window[Window("sliding", 20)]].shape[0] == 3


def test_a_state_slot_that_is_used_again_starts_at_zero(folders):
    eng = host_engine(folders["S"], 128, max_requests=1)
    reqs = requests_for(folders["S"], (30, 25), 60)
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": reqs["r0"], "want": [29]}], "end": ["r0"]},
             {"step": 1, "entries": [{"id": "r1", "tokens": reqs["r1"][:10], "want": [9]}], "end": []},
             {"step": 2, "entries": [{"id": "r1", "tokens": reqs["r1"][10:], "want": [0, 14]}], "end": ["r1"]}]
    S.compare_with_plain(H.run_steps(eng, steps), folders["S"], reqs, 2e-5)


def test_trace_replay_on_the_host(folders, tmp_path):
    from spite_b200.engine.trace import replay
    folder = folders["P"]
    reqs = requests_for(folder, (50, 21, 5), 70)
    steps = H.steps_mixed(reqs, {r: len(t) - 4 for r, t in reqs.items()}, seed=9)
    eng = host_engine(folder, H.max_tokens_of(steps), page_size=64)
    log = io.StringIO()
    replay(eng, [json.dumps(s) for s in steps], tmp_path / "out", log=log)
    assert log.getvalue().split("\n")[:-1] == [f"done {s['step']}" for s in steps]
    pos, got = {}, {}
    for s in steps:
        rows = np.fromfile(tmp_path / "out" / f"{s['step']}.f32", dtype="<f4").reshape(-1, S.CONFIG_P["vocab"])
        i = 0
        for e in s["entries"]:
            base = pos.get(e["id"], 0)
            for w in e["want"]:
                got[(e["id"], base + w)] = torch.from_numpy(rows[i].copy())
                i += 1
            pos[e["id"]] = base + len(e["tokens"])
    S.compare_with_plain(got, folder, reqs, 2e-5)
