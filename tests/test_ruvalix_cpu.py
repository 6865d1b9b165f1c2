"""Ruvalix on the CPU: the plain model's mechanisms one by one, and the engine (configuration,
loader, run order, pages and states, step function, scheduler) over the kernels' plain
references against the plain model."""
import json
import math
import os

import numpy as np
import pytest
import torch

from garuda_b200 import Engine, SamplingParams, StepEntry, ConfigError, WeightError
from garuda_b200.config.registry import build_model, read_model_config
from garuda_b200.parts.base import FixedState, PagedKV
from tests import helpers
from tests.plain import ruvalix_plain as rp
from tests.plain.cpu_ops import CpuOps
from tests.ruvalix_cases import CASES, RA, RB, RD, edge_model, model_dir, plain_logits, random_tokens, weights


def assert_close(got, want, dtype, what):
    """Against the 64-bit plain model, as a fraction of the largest logit: 32-bit sums in another
    order through up to eight layer runs with sharpened weights."""
    scale = max(float(np.abs(want).max()), 1e-6)
    err = float(np.abs(np.asarray(got) - want).max())
    assert got.shape == want.shape and np.isfinite(got).all(), what
    helpers.OBSERVED[f"ruvalix/{dtype}"] = max(helpers.OBSERVED.get(f"ruvalix/{dtype}", 0.0), err / scale)
    assert err <= 5e-5 * scale, f"{what}: max difference {err:.3e} (limit {5e-5 * scale:.3e})"


def engine(name, **kw):
    kw.setdefault("page_size", 8)
    kw.setdefault("kv_tokens", 512)
    kw.setdefault("context", 256)
    return Engine(model_dir(name), dtype="float32", ops=CpuOps(), cuda_graphs=False, **kw)


# ------------------------------------------------------------------ the plain model's mechanisms
def test_norm_adds_one_to_its_weight_and_has_eps_inside_the_root():
    assert np.allclose(rp.offset_norm(np.array([[2.0, 2.0]]), np.array([0.5, -1.0]), 5.0), [[1.0, 0.0]])


def test_gates_are_capped_and_the_forget_gate_is_a_log_sigmoid():
    assert np.allclose(rp.soft_cap(np.array([0.0, 3.0, 1e6]), 3.0), [0.0, 3 * math.tanh(1.0), 3.0])
    z = np.array([-700.0, 0.0, 2.0])
    assert np.allclose(rp.log_sigmoid(z), [-700.0, -math.log(2.0), -math.log1p(math.exp(-2.0))])


def test_matrix_memory_by_hand():
    """Two tokens. The running maximum starts at zero, so a first input gate of -3 is not brought up to one."""
    q, k, v = np.array([[2.0, 0.0], [1.0, 1.0]]), np.array([[1.0, 3.0], [2.0, 0.0]]), np.array([[5.0], [7.0]])
    i, f = np.array([-3.0, 1.0]), np.array([-0.5, -0.25])
    out = rp.matrix_memory(q, k, v, i, f)
    m1 = max(-0.5 + 0.0, -3.0)
    s1, n1 = math.exp(-3.0 - m1) * np.array([1.0, 3.0]) * 5.0, math.exp(-3.0 - m1) * np.array([1.0, 3.0])
    assert np.allclose(out[0], 2.0 * s1[0] / (max(abs(2.0 * n1[0]), math.exp(-m1)) + 1e-6))        # the floor exp(-m) is what counts
    assert abs(2.0 * n1[0]) < math.exp(-m1)
    m2 = max(-0.25 + m1, 1.0)
    keep, put = math.exp(-0.25 + m1 - m2), math.exp(1.0 - m2)
    s2, n2 = keep * s1 + put * np.array([2.0, 0.0]) * 7.0, keep * n1 + put * np.array([2.0, 0.0])
    assert np.allclose(out[1], s2.sum() / (max(abs(n2.sum()), math.exp(-m2)) + 1e-6))


def test_matrix_memory_without_its_running_maximum():
    """The memory relative to exp(m) is the memory: the same read-out from the unscaled recurrence with a floor of one."""
    rng = np.random.default_rng(0)
    T, D, P = 30, 5, 4
    q, k, v = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, P))
    i, f = rng.uniform(-2, 2, T), rng.uniform(-1, 0, T)
    S, n, want = np.zeros((D, P)), np.zeros(D), np.zeros((T, P))
    for t in range(T):
        S, n = math.exp(f[t]) * S + math.exp(i[t]) * np.outer(k[t], v[t]), math.exp(f[t]) * n + math.exp(i[t]) * k[t]
        want[t] = (q[t] @ S) / max(abs(n @ q[t]), 1.0)
    assert np.allclose(rp.matrix_memory(q, k, v, i, f), want, rtol=1e-4)


def test_stretched_frequencies_by_hand():
    freq, factor = rp.yarn(100.0, 8, {"factor": 4.0, "original": 64, "fast": 5.0, "slow": 1.0})
    base = 100.0 ** (-np.arange(4) / 4.0)
    lo = max(math.floor(8 * math.log(64 / (10 * math.pi)) / (2 * math.log(100.0))), 0)
    hi = min(math.ceil(8 * math.log(64 / (2 * math.pi)) / (2 * math.log(100.0))), 7)
    assert (lo, hi) == (0, 3)
    ramp = np.array([0.0, 1 / 3, 2 / 3, 1.0])
    assert np.allclose(freq, base * (1 - ramp) + base / 4 * ramp) and np.isclose(factor, 0.1 * math.log(4.0) + 1)
    from garuda_b200.parts.rotary import stretched_frequencies
    for dims, base, s in ((8, 100.0, (4.0, 64, 5.0, 1.0)), (24, 5e5, (2.0, 2000, 30.0, 1.0)), (6, 50.0, (3.0, 10, 9.0, 8.0)), (64, 1e4, (16.0, 4096, 32.0, 0.5))):
        scaling = dict(zip(("factor", "original", "fast", "slow"), s))
        (a, fa), (b, fb) = rp.yarn(base, dims, scaling), stretched_frequencies(base, dims, scaling)
        assert np.allclose(a, b, rtol=1e-14) and np.isclose(fa, fb)


def test_rotation_pairs_halves_of_the_first_channels_and_leaves_the_rest():
    x = np.arange(1.0, 8.0)[None, None, :]
    y = rp.rotate_half(x, [3], np.array([0.5, 0.1]), 2.0)[0, 0]
    for i, f in ((0, 0.5), (1, 0.1)):
        u, v = x[0, 0, i], x[0, 0, i + 2]
        assert np.isclose(y[i], 2 * (u * math.cos(3 * f) - v * math.sin(3 * f))) and np.isclose(y[i + 2], 2 * (v * math.cos(3 * f) + u * math.sin(3 * f)))
    assert np.allclose(y[4:], x[0, 0, 4:])


def test_window_counts_the_position_itself():
    m = rp.window_mask(6, 3)
    assert [np.flatnonzero(r).tolist() for r in m] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4], [3, 4, 5]]
    assert rp.window_mask(3, None).tolist() == np.tril(np.ones((3, 3), bool)).tolist()


def test_the_second_map_is_taken_off_and_the_difference_normed():
    W = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.1]), "lq2": np.array([1.0, 0.0]), "lk2": np.array([0.2, 9.0])}
    lam = rp.mixing_number(W, "", 0.3)
    assert np.isclose(lam, math.exp(0.7) - math.exp(0.2) + 0.3)
    a1, a2 = np.array([[3.0, 1.0]]), np.array([[1.0, 1.0]])
    d = np.array([3.0 - lam, 1.0 - lam])
    assert np.allclose(rp.difference_of_maps(a1, a2, lam, 0.3, 0.0), 0.7 * d / np.sqrt(np.mean(d * d)))


def test_choice_goes_by_corrected_scores_within_the_best_groups():
    s = np.array([0.30, 0.20, 0.10, 0.15, 0.05, 0.20])
    none = np.zeros(6)
    assert rp.choose(s, none, 2, 1, 1).tolist() == [0, 1]
    assert rp.choose(s, np.array([0, 0, 0, 0.2, 0, 0]), 2, 1, 1).tolist() == [3, 0]
    assert rp.choose(s, none, 2, 3, 1).tolist() == [0, 1]               # groups 0-1, 2-3, 4-5: the best is the first
    assert rp.choose(s, none, 3, 3, 2).tolist() == [0, 1, 5]
    # every choice score negative: what lies outside the kept group must not win with a zero
    assert rp.choose(s, np.full(6, -1.0), 2, 3, 1).tolist() == [0, 1]


def test_experts_that_return_their_input_and_weights_without_the_correction():
    d = 2
    W = {"router": np.array([[1.0, 0], [0, 1.0], [0.5, 0.5]]), "correction": np.array([-9.0, 0.0, 0.0]), "shared.gate": np.eye(d), "shared.up": np.eye(d),
         "shared.down": np.eye(d)}
    for e in range(2):
        W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"] = np.eye(d), np.eye(d) * 10, np.eye(d) * (e + 1)
    f = {"router": {"experts": 2, "top": 2, "identity": 1}, "shared": {"ff": 2}}
    h = np.array([[2.0, 1.0]])
    s = np.exp([2.0, 1.0, 1.5]) / np.exp([2.0, 1.0, 1.5]).sum()
    silu = lambda z: z / (1 + np.exp(-z))
    want = s[1] * 2 * silu(h) * 10 * h + s[2] * h + silu(h) * h            # expert 0 is never chosen; shares not renormalized
    assert np.allclose(rp.routed_ff(W, "", f, h), want)


def test_passes_of_the_loop():
    assert rp.run_order(RA) == [(0, None), (1, 0), (2, None), (1, 1), (2, None)]
    toks, W = random_tokens("RA", 9, 8), {n: np.asarray(a, dtype=np.float64) for n, a in weights("RA").items()}
    seen = []
    rp.forward(RA, W, toks, seen)
    x0 = rp.offset_norm(W["embed"][toks], W["embed.norm"], 1e-5)
    x = np.concatenate([seen[2], x0], -1) @ W["loop.in"].T + W["loop.step"][1]             # before the second pass
    p, c = "l1.", RA["layers"][1]
    x = x + rp.offset_norm(rp.attention(W, p + "mix.", c["mixer"], 1e-5, rp.offset_norm(x, W[p + "norm1"], 1e-5)), W[p + "norm1b"], 1e-5)
    x = x + rp.offset_norm(rp.routed_ff(W, p + "mlp.", c["mlp"], rp.offset_norm(x, W[p + "norm2"], 1e-5)), W[p + "norm2b"], 1e-5)
    assert np.allclose(seen[3], x)


# ------------------------------------------------------------------ configuration, tensors, cache needs
def test_configuration_errors_name_the_key():
    def broken(change):
        cfg = json.loads(json.dumps(RB))
        change(cfg)
        return cfg
    cases = [(lambda c: c.pop("norm"), "eps"), (lambda c: c["layers"][0]["mixer"].pop("diff"), "layers[0].mixer.diff"),
             (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "layers[0].mixer.heads"),
             (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "layers[0].mixer.mask.size"),
             (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=34), "layers[0].mixer.rot.dims"),
             (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "layers[0].mixer.rot.dims"),
             (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "layers[0].mixer.rot.scaling.slow"),
             (lambda c: c["layers"][0]["mlp"]["router"].update(groups={"count": 3, "keep": 1}), "layers[0].mlp.router.groups"),
             (lambda c: c["layers"][0]["mlp"]["router"]["groups"].pop("keep"), "layers[0].mlp.router.groups.keep"),
             (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "layers[0].mlp.router.top"),
             (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "layers[0].mlp.kind"),
             (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "layers[0].mlp.shared.ff"),
             (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "layers[1].mixer.gate_cap"),
             (lambda c: c["layers"][1].update(type="gru"), "layers[1].type"),
             (lambda c: c["loop"].update(stop=5), "loop"), (lambda c: c["loop"].pop("times"), "loop.times")]
    for change, key in cases:
        with pytest.raises(ConfigError, match=key.replace("[", r"\[").replace("]", r"\]")):
            read_model_config(broken(change))


def test_run_order_and_cache_needs_come_from_the_configuration():
    _, model = build_model(RB)
    assert [c.layer for c in model.spec.order] == [0, 1, 0, 1, 0, 1, 2, 3]
    assert [c.mix_embedding is not None for c in model.spec.order] == [True, False] * 3 + [False, False]
    assert [c.add_row for c in model.spec.order][::2] == [("loop.step", 0), ("loop.step", 1), ("loop.step", 2), None]
    # a pass has a cache or a state of its own; layers of unlike windows have page groups of their own
    assert {g.need: g.calls for g in model.cache_groups} == {PagedKV(2, 64, 40, value_dim=64): (0, 2, 4), PagedKV(2, 32, 100, value_dim=16): (6,)}
    assert model.state_calls == [1, 3, 5, 7] and model.need_at(1) == FixedState((2 * 64 * 32 + 2 * 64 + 2 + 2,))
    names = set(model.expected_tensors())
    assert {"embed.norm", "loop.in", "loop.step", "l0.norm1b", "l0.norm2b", "l0.mix.q.b", "l0.mix.lk2", "l0.mix.g", "l1.mix.i.b", "l1.mix.norm",
            "l0.mlp.correction", "l0.mlp.shared.down", "l3.mlp.e5.gate", "final.norm", "head"} <= names
    assert not {"l1.mlp.shared.up", "l0.mlp.e6.up", "l3.mlp.e6.gate", "l0.mix.o.b", "l0.mix.g.b"} & names
    assert model.expected_tensors()["l0.mlp.router"].shape == (8, 128) and model.expected_tensors()["l3.mlp.router"].shape == (12, 128)
    _, model = build_model(RA)
    assert model.need_at(0) == FixedState(((3 * 7 * 11 + 21 + 3 + 3) // 4 * 4,)) and "l2.norm2" not in model.expected_tensors()


def test_a_missing_and_an_unexpected_tensor_are_reported(tmp_path):
    from garuda_b200.weights import SafetensorsFolder, write_safetensors
    f = SafetensorsFolder(model_dir("RA"))
    tensors = {n: f.tensor(n) for n in f.names() if n not in ("l1.mix.lq1", "loop.in")}
    tensors["l1.mlp.e4.up"] = torch.zeros(18, 44)
    os.makedirs(tmp_path / "m")
    write_safetensors(str(tmp_path / "m" / "model.safetensors"), tensors)
    (tmp_path / "m" / "config.json").write_text(json.dumps(RA))
    with pytest.raises(WeightError) as e:
        Engine(str(tmp_path / "m"), dtype="float32", ops=CpuOps(), cuda_graphs=False)
    assert all(n in str(e.value) for n in ("l1.mix.lq1", "loop.in", "l1.mlp.e4.up"))


# ------------------------------------------------------------------ the engine against the plain model
@pytest.mark.parametrize("name", ["RA", "RB", "RC", "RD"])
def test_whole_prompt(name):
    toks = random_tokens(name, 45, 2)
    e = engine(name)
    got = e.step([StepEntry(1, toks, range(len(toks)))]).numpy()
    assert_close(got, plain_logits(name, torch.float32, toks), "float32", f"{name} whole")


@pytest.mark.parametrize("name", ["RA", "RB"])
def test_the_residual_after_every_layer(name):
    toks = random_tokens(name, 20, 6)
    e = engine(name)
    seen = []
    e.runner.layer_probe = lambda i, x: seen.append(x.clone().numpy())
    e.step([StepEntry(1, toks, [])])
    want = []
    rp.forward(CASES[name][0], weights(name), toks, want)
    assert len(seen) == len(want) == len(rp.run_order(CASES[name][0]))
    for i, (a, b) in enumerate(zip(seen, want)):
        assert np.abs(a - b).max() <= 5e-5 * np.abs(b).max(), f"layer run {i}"


@pytest.mark.parametrize("name", ["RA", "RD"])
def test_token_by_token_from_the_first_token(name):
    toks = random_tokens(name, 40, 3)
    e = engine(name)
    got = np.stack([e.step([StepEntry(1, [t], [0])]).numpy()[0].copy() for t in toks])
    assert_close(got, plain_logits(name, torch.float32, toks), "float32", f"{name} token by token")


@pytest.mark.parametrize("name,cuts", [("RA", [2, 4, 5, 12, 13, 16, 24, 33, 35, 50]), ("RB", [1, 3, 8, 9, 17, 40, 50]),
                                       ("RD", [7, 9, 11, 26, 28, 33, 35, 50])])
def test_portions_cut_anywhere(name, cuts):
    toks = random_tokens(name, 50, 4)
    e = engine(name)
    rows, a = [], 0
    for b in cuts:
        rows.append(e.step([StepEntry(1, toks[a:b], range(b - a))]).numpy().copy())
        a = b
    assert_close(np.concatenate(rows), plain_logits(name, torch.float32, toks), "float32", f"{name} in portions")


def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again():
    name = "RA"
    e = engine(name, kv_tokens=136, max_concurrent=3)          # 17 pages of 8 for three requests of up to 60 tokens
    prompts = {i: random_tokens(name, n, 10 + i) for i, n in enumerate([60, 23, 41, 9, 37, 52])}
    at = {i: 0 for i in prompts}
    got = {i: [] for i in prompts}
    live, waiting = [], list(prompts)
    rng = np.random.default_rng(0)
    while live or waiting:
        while waiting and len(live) < 3 and sum(-(-len(prompts[i]) // 8) for i in live + waiting[:1]) <= 17:
            live.append(waiting.pop(0))
        entries = []
        for i in live:
            n = int(rng.choice([1, 1, 2, 3, 7, 16]))
            n = min(n, len(prompts[i]) - at[i])
            entries.append(StepEntry(100 + i, prompts[i][at[i]:at[i] + n], range(n)))
        out = e.step(entries).numpy()
        row = 0
        for i, en in zip(list(live), entries):
            n = len(en.tokens)
            got[i].append(out[row:row + n].copy())
            row += n
            at[i] += n
            if at[i] == len(prompts[i]):
                e.runner.end(100 + i)
                live.remove(i)
        e.cache.manager.check_invariants()
    assert e.cache.manager.pages_reused > 0
    for i, toks in prompts.items():
        assert_close(np.concatenate(got[i]), plain_logits(name, torch.float32, toks), "float32", f"request {i} in a mixed batch")


def test_a_slot_used_again_starts_from_zero_state():
    name = "RD"
    e = engine(name, max_concurrent=1)
    a, b = random_tokens(name, 30, 40), random_tokens(name, 17, 41)
    e.step([StepEntry(1, a, [])])
    e.runner.end(1)
    got = e.step([StepEntry(2, b, range(len(b)))]).numpy()
    assert_close(got, plain_logits(name, torch.float32, b), "float32", "the second user of a slot")


def test_long_decoding_after_a_prompt():
    name = "RA"
    toks = random_tokens(name, 120, 7)
    e = engine(name)
    rows = [e.step([StepEntry(1, toks[:20], range(20))]).numpy().copy()]
    rows += [e.step([StepEntry(1, [t], [0])]).numpy().copy() for t in toks[20:]]
    assert_close(np.concatenate(rows), plain_logits(name, torch.float32, toks), "float32", "100 decoded tokens")


def test_a_key_just_inside_and_just_outside_the_window(tmp_path):
    """Token 0 once, 39 (the last seen) and 40 (the first not seen) positions in front of a query for it, in a prompt and decoded."""
    d, cfg = edge_model(str(tmp_path / "m"), torch.float32, window=40)
    W = helpers.folder_weights(d)
    base = np.random.default_rng(5).integers(2, 80, 70)
    for back, seen in ((39, True), (40, False)):
        toks = base.copy()
        toks[60], toks[60 - back] = 1, 0
        ref = rp.forward(cfg, W, toks)
        other = base.copy()
        other[60] = 1
        change = np.abs(rp.forward(cfg, W, other)[60] - ref[60]).max() / np.abs(ref[60]).max()
        assert change > 0.2 if seen else change == 0.0
        toks = toks.tolist()
        e = Engine(d, dtype="float32", ops=CpuOps(), cuda_graphs=False, page_size=8, kv_tokens=256, context=128)
        whole = e.step([StepEntry(1, toks, range(70))]).numpy().copy()
        assert_close(whole, ref.astype(np.float32), "float32", f"{back} back, whole")
        e.step([StepEntry(2, toks[:58], [])])
        dec = np.concatenate([e.step([StepEntry(2, [t], [0])]).numpy().copy() for t in toks[58:]])
        assert_close(dec, ref[58:].astype(np.float32), "float32", f"{back} back, decoded")


def test_greedy_generation_through_the_scheduler():
    name = "RA"
    e = engine(name, max_batch_tokens=16, prefill_chunk=8)
    prompts = [random_tokens(name, n, 20 + n) for n in (19, 5, 30)]
    results = e.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12))
    for p, r in zip(prompts, results):
        seq = list(p)
        for _ in range(12):
            seq.append(int(np.argmax(rp.forward(RA, weights(name), seq)[-1])))
        assert r.tokens == seq[len(p):]
        assert len(set(r.tokens)) > 2


def test_parts_refuse_what_they_do_not_know():
    from garuda_b200.parts import DifferentialAttention, MatrixMemory, Rotary, RoutedExperts
    with pytest.raises(ValueError, match="groups"):
        RoutedExperts(16, 5, 2, 8, groups=(3, 1))
    with pytest.raises(ValueError, match="uses 1 to 2"):
        RoutedExperts(16, 6, 3, 8, groups=(3, 1))
    with pytest.raises(ValueError, match="correction"):
        RoutedExperts(16, 4, 2, 8, correction=True)
    with pytest.raises(ValueError, match="return their input"):
        RoutedExperts(16, 4, 2, 8, identity=1, scale_input=True)
    with pytest.raises(ValueError, match="multiple"):
        DifferentialAttention(16, 3, 2, 8)
    with pytest.raises(ValueError, match="positive"):
        MatrixMemory(16, 2, 8, 8, 0.0, 1e-5)
    with pytest.raises(ValueError, match="covers the head"):
        Rotary(1e4, 16, rotary_dim=8, scaling=dict(factor=2.0, original=100, fast=8.0, slow=1.0))


def test_a_stream_mixed_with_a_plain_embedding():
    """The mix before a pass in a model whose embedding is scaled, not normed, and whose layers are pre-norm ones."""
    from dataclasses import replace
    from garuda_b200.cache.manager import CacheConfig, PagedCache
    from garuda_b200.engine.step import StepRunner
    from garuda_b200.models.decoder import Decoder
    from garuda_b200.models.ruvalix import ruvalix_spec
    toks, W = random_tokens("RA", 11, 6), {n: np.asarray(a, dtype=np.float64) for n, a in weights("RA").items()}
    spec = ruvalix_spec(read_model_config(RA))
    spec.layers = [replace(spec.layers[2], arrangement="pre_norm")]
    spec.order, spec.embedding_norm, spec.embedding_scale = [replace(c, layer=0) for c in (spec.order[1], spec.order[3])], None, 2.0
    model, ops = Decoder(spec), CpuOps()
    model.load({n: torch.tensor(np.asarray(weights("RA")[n])) for n in model.expected_tensors()}, ops, torch.float32)
    cache = PagedCache(model, CacheConfig(page_size=8, max_tokens=64, max_positions=64), torch.float32, "cpu")
    runner, seen = StepRunner(model, cache, ops, torch.float32, "cpu"), []
    runner.layer_probe = lambda i, x: seen.append(x.clone().numpy())
    cache.acquire(1)
    runner.run([StepEntry(1, toks, [])])
    x = x0 = W["embed"][toks] * 2.0
    for t in range(2):
        x = np.concatenate([x, x0], -1) @ W["loop.in"].T + W["loop.step"][t]
        x = x + rp.mlstm(W, "l2.mix.", RA["layers"][2]["mixer"], 1e-5, rp.offset_norm(x, W["l2.norm1"], 1e-5))
        assert np.abs(seen[t] - x).max() <= 2e-5 * np.abs(x).max()
