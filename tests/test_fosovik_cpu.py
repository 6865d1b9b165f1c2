"""Fosovik on the CPU: the plain model's mechanisms one by one, and the engine (configuration,
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
from tests.fosovik_cases import CASES, FA, FB, FC, FD, model_dir, plain_logits, random_tokens, weights
from tests.plain import fosovik_plain as fp
from tests.plain.cpu_ops import CpuOps


def assert_close(got, want, dtype, what):
    """Against the 64-bit plain model, as a fraction of the largest logit: 32-bit sums in another
    order through up to six layers with sharpened weights."""
    scale = max(float(np.abs(want).max()), 1e-6)
    err = float(np.abs(np.asarray(got) - want).max())
    assert got.shape == want.shape and np.isfinite(got).all(), what
    helpers.OBSERVED[f"fosovik/{dtype}"] = max(helpers.OBSERVED.get(f"fosovik/{dtype}", 0.0), err / scale)
    assert err <= 5e-5 * scale, f"{what}: max difference {err:.3e} (limit {5e-5 * scale:.3e})"


def engine(name, **kw):
    kw.setdefault("page_size", 8)
    kw.setdefault("kv_tokens", 512)
    kw.setdefault("context", 256)
    return Engine(model_dir(name), dtype="float32", ops=CpuOps(), cuda_graphs=False, **kw)


# ------------------------------------------------------------------ the plain model's mechanisms
def test_norm_has_no_statistics():
    W = {"n": np.array([2.0, 3.0]), "n.b": np.array([0.5, -1.0]), "n.alpha": np.array(0.5)}
    v = np.array([[1.0, 4.0]])
    assert np.allclose(fp.squash(v, W, "n"), [[2 * math.tanh(0.5) + 0.5, 3 * math.tanh(2.0) - 1.0]])


def test_unit_rms_has_eps_inside_the_root():
    assert np.allclose(fp.unit_rms(np.array([[3.0, 4.0]]), 0.0), np.array([[3.0, 4.0]]) / np.sqrt(12.5))
    assert np.allclose(fp.unit_rms(np.array([[2.0, 2.0]]), 5.0), [[2.0 / 3.0, 2.0 / 3.0]])


def test_queries_grow_in_steps_that_start_one_position_early():
    f = fp.query_factor(np.arange(0, 20), 0.5, 9)
    assert np.allclose(f[:8], 1.0)                                       # positions 0..7: floor((p + 1) / 9) = 0
    assert np.allclose(f[8:17], 1 + 0.5 * np.log(2)) and np.allclose(f[17:], 1 + 0.5 * np.log(3))


def test_sink_counts_once_unscaled_and_has_no_value():
    s = np.array([[0.0, np.log(2.0), -np.inf]])
    assert np.allclose(fp.softmax_sink(s, np.log(5.0)), [[1 / 8, 2 / 8, 0.0]])


def test_gelu_is_the_exact_one():
    z = np.array([1.0, -2.0, 0.0])
    assert np.allclose(fp.gelu_erf(z), [0.8413447460685429, -2 * 0.022750131948179212, 0.0])


def test_short_convolution_is_causal_starts_from_zeros_and_has_a_bias():
    x = np.arange(1.0, 6.0)[:, None] * np.array([[1.0, 10.0]])
    taps = np.array([[0.5, 0.0, 2.0], [0.0, 1.0, 0.0]])                # the last column weighs the current token
    y = fp.causal_conv(x, taps, np.array([100.0, 0.0]))
    assert np.allclose(y[:, 0], [102.0, 104.0, 106.5, 109.0, 111.5]) and np.allclose(y[:, 1], [0.0, 10.0, 20.0, 30.0, 40.0])


def test_state_space_by_hand():
    x, B, C = np.array([[2.0], [3.0]]), np.array([[1.0, 0.0], [1.0, 2.0]]), np.array([[5.0, 7.0], [1.0, 1.0]])
    dt, rate, D = np.array([0.5, 0.25]), 2.0, 10.0
    y = fp.state_space(x, B, C, dt, rate, D)
    s0 = np.array([1.0, 0.0])                                            # dt B x
    s1 = math.exp(-0.5) * s0 + 0.25 * 3.0 * np.array([1.0, 2.0])
    assert np.allclose(y[:, 0], [5.0 * s0[0] + 20.0, s1.sum() + 30.0])


def test_grouped_norm_takes_each_part_by_itself():
    v = np.array([[1.0, 1.0, 10.0, 10.0]])
    assert np.allclose(fp.grouped_rms(v, 2, 0.0), [[1, 1, 1, 1]]) and not np.allclose(fp.grouped_rms(v, 1, 0.0), 1.0)


def test_gated_feed_forward_clamps_only_as_written():
    W = {"gate": np.array([[1.0]]), "up": np.array([[1.0]]), "down": np.array([[1.0]])}
    for h, g, u in ((5.0, 1.5, 1.5), (-5.0, -5.0, -1.5), (0.5, 0.5, 0.5)):       # the gate is clamped from above alone
        want = g / (1 + math.exp(-1.702 * g)) * (u + 1)
        assert np.allclose(fp.dense_ff(W, "", 1.5, np.array([[h]])), want)


def test_router_weighs_by_the_softmax_over_all_experts_not_renormalized():
    d = 3
    W = {"router": np.array([[2.0, 0, 0], [1.0, 0, 0], [0.0, 0, 0]])}
    for e in range(3):
        W[f"e{e}.up"], W[f"e{e}.down"] = np.eye(d) * 10, np.eye(d) * (e + 1)
    s = np.exp([2.0, 1.0, 0.0]) / np.exp([2.0, 1.0, 0.0]).sum()
    assert np.allclose(fp.routed_ff(W, "", 2, np.array([[1.0, 0.0, 0.0]]))[0, 0], 10.0 * (s[0] * 1 + s[1] * 2))


def test_both_sublayers_read_the_same_norm():
    """Layer 1 of the second configuration: its output is the sum of both sublayers of one normed input."""
    toks = random_tokens("FB", 12, 8)
    W = {n: np.asarray(a, dtype=np.float64) for n, a in weights("FB").items()}
    seen = []
    fp.forward(FB, W, toks, seen)
    h = fp.squash(seen[0], W, "l1.norm1")
    m, f = FB["layers"][1]["mixer"], FB["layers"][1]["mlp"]
    want = seen[0] + fp.mamba2(W, "l1.mix.", m, 1e-6, h) + fp.routed_ff(W, "l1.mlp.", f["router"]["top"], h)
    assert np.allclose(seen[1], want)


# ------------------------------------------------------------------ configuration, tensors, cache needs
def test_configuration_errors_name_the_key():
    def broken(change):
        cfg = json.loads(json.dumps(FB))
        change(cfg)
        return cfg
    cases = [(lambda c: c.pop("norm"), "eps"), (lambda c: c["layers"][0]["mixer"].pop("kv_heads"), "layers[0].mixer.kv_heads"),
             (lambda c: c["layers"][0]["mixer"]["q_temp"].pop("every"), "layers[0].mixer.q_temp.every"),
             (lambda c: c["layers"][0]["mlp"]["router"].pop("top"), "layers[0].mlp.router.top"),
             (lambda c: c["layers"][1]["mixer"].pop("state"), "layers[1].mixer.state"),
             (lambda c: c["layers"][1]["mixer"].update(conv=0), "layers[1].mixer.conv"),
             (lambda c: c["layers"][1]["mixer"].update(groups=3), "layers[1].mixer.groups"),
             (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "norm_groups"),
             (lambda c: c["layers"][2]["mlp"].pop("limit"), "layers[2].mlp.limit"),
             (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "layers[2].mixer.kv_from"),
             (lambda c: c["layers"][2]["mixer"].update(kv_from=4), "layers[2].mixer.kv_from"),
             (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "layers[4].mixer.kv_from"),
             (lambda c: c["layers"][2]["mixer"].update(dim=32), "layers[2].mixer"),
             (lambda c: c["layers"][3].update(type="window"), "layers[3].type"),
             (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "layers[0].mlp.kind")]
    for change, key in cases:
        with pytest.raises(ConfigError, match=key.replace("[", r"\[").replace("]", r"\]")):
            read_model_config(broken(change))


def test_run_order_and_cache_needs_come_from_the_configuration():
    _, model = build_model(FA)
    assert [c.reads_cache_of for c in model.spec.order] == [None, None, 1, None, None]
    assert {g.need: g.calls for g in model.cache_groups} == {PagedKV(2, 12, None, value_dim=20): (1,)}
    assert model.need_at(0) == FixedState((6 * 9 * 10 + 2 * (54 + 60),)) and model.need_at(3) == FixedState((2 * 20 * 7,))
    names = set(model.expected_tensors())
    assert {"l0.norm1.alpha", "l0.mix.conv.b", "l0.mlp.e4.up", "l1.mix.sink", "l2.mix.sink", "l2.mix.q", "final.norm.b", "head"} <= names
    assert not {"l2.mix.k", "l2.mix.v", "l0.mlp.e0.gate", "l0.norm2", "l3.mlp.up"} & names
    _, model = build_model(FB)
    assert [c.reads_cache_of for c in model.spec.order] == [None, None, 0, None, 0, None]


def test_a_missing_and_an_unexpected_tensor_are_reported(tmp_path):
    from garuda_b200.weights import SafetensorsFolder, write_safetensors
    f = SafetensorsFolder(model_dir("FA"))
    tensors = {n: f.tensor(n) for n in f.names() if n != "l2.mix.sink"}
    tensors["l2.mix.k"] = torch.zeros(24, 44)
    os.makedirs(tmp_path / "m")
    write_safetensors(str(tmp_path / "m" / "model.safetensors"), tensors)
    (tmp_path / "m" / "config.json").write_text(json.dumps(FA))
    with pytest.raises(WeightError) as e:
        Engine(str(tmp_path / "m"), dtype="float32", ops=CpuOps(), cuda_graphs=False)
    assert "l2.mix.sink" in str(e.value) and "l2.mix.k" in str(e.value)


def test_a_layer_that_reads_anothers_keys_holds_no_pages():
    e = engine("FB")
    assert len(e.cache.groups) == 1 and e.cache.k_pools[0].shape[0] == 1      # one call's pages for three attention layers


# ------------------------------------------------------------------ the engine against the plain model
@pytest.mark.parametrize("name", ["FA", "FB", "FC", "FD"])
def test_whole_prompt(name):
    toks = random_tokens(name, 45, 2)
    e = engine(name)
    got = e.step([StepEntry(1, toks, range(len(toks)))]).numpy()
    assert_close(got, plain_logits(name, torch.float32, toks), "float32", f"{name} whole")


@pytest.mark.parametrize("name", ["FA", "FD"])
def test_the_residual_after_every_layer(name):
    toks = random_tokens(name, 20, 6)
    e = engine(name)
    seen = []
    e.runner.layer_probe = lambda i, x: seen.append(x.clone().numpy())
    e.step([StepEntry(1, toks, [])])
    want = []
    fp.forward(CASES[name][0], weights(name), toks, want)
    assert len(seen) == len(want) == len(CASES[name][0]["layers"])
    for i, (a, b) in enumerate(zip(seen, want)):
        assert np.abs(a - b).max() <= 2e-5 * np.abs(b).max(), f"layer {i}"


@pytest.mark.parametrize("name", ["FA", "FD"])
def test_token_by_token_from_the_first_token(name):
    toks = random_tokens(name, 40, 3)
    e = engine(name)
    got = np.stack([e.step([StepEntry(1, [t], [0])]).numpy()[0].copy() for t in toks])
    assert_close(got, plain_logits(name, torch.float32, toks), "float32", f"{name} token by token")


@pytest.mark.parametrize("name,cuts", [("FA", [2, 4, 5, 12, 13, 16, 24, 33, 35, 50]), ("FB", [1, 3, 8, 9, 17, 40, 50]),
                                       ("FD", [7, 9, 11, 26, 28, 33, 35, 50])])
def test_portions_cut_anywhere(name, cuts):
    toks = random_tokens(name, 50, 4)
    e = engine(name)
    rows, a = [], 0
    for b in cuts:
        rows.append(e.step([StepEntry(1, toks[a:b], range(b - a))]).numpy().copy())
        a = b
    assert_close(np.concatenate(rows), plain_logits(name, torch.float32, toks), "float32", f"{name} in portions")


def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again():
    name = "FA"
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
    name = "FD"
    e = engine(name, max_concurrent=1)
    a, b = random_tokens(name, 30, 40), random_tokens(name, 17, 41)
    e.step([StepEntry(1, a, [])])
    e.runner.end(1)
    got = e.step([StepEntry(2, b, range(len(b)))]).numpy()
    assert_close(got, plain_logits(name, torch.float32, b), "float32", "the second user of a slot")


def test_long_decoding_after_a_prompt():
    name = "FA"
    toks = random_tokens(name, 120, 7)
    e = engine(name)
    rows = [e.step([StepEntry(1, toks[:20], range(20))]).numpy().copy()]
    rows += [e.step([StepEntry(1, [t], [0])]).numpy().copy() for t in toks[20:]]
    assert_close(np.concatenate(rows), plain_logits(name, torch.float32, toks), "float32", "100 decoded tokens")


def test_greedy_generation_through_the_scheduler():
    name = "FA"
    e = engine(name, max_batch_tokens=16, prefill_chunk=8)
    prompts = [random_tokens(name, n, 20 + n) for n in (19, 5, 30)]
    results = e.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12))
    for p, r in zip(prompts, results):
        seq = list(p)
        for _ in range(12):
            seq.append(int(np.argmax(fp.forward(FA, weights(name), seq)[-1])))
        assert r.tokens == seq[len(p):]
        assert len(set(r.tokens)) > 2


def test_plain_experts_refuse_what_they_do_not_know():
    from garuda_b200.parts import RoutedExperts
    for kw in (dict(activation="clamped_swish"), dict(activation="gelu", shared_inner=8)):
        with pytest.raises(ValueError, match="without a gate"):
            RoutedExperts(16, 4, 2, 8, gated=False, **kw)


def test_parallel_layers_take_a_multiplier():
    """x + m (mixer(h) + ff(h)), through parts that scale as they add."""
    from garuda_b200.models.fosovik import fosovik_spec
    from garuda_b200.models.decoder import Decoder
    from garuda_b200.cache.manager import CacheConfig, PagedCache
    from garuda_b200.engine.step import StepRunner
    from dataclasses import replace
    toks, W = random_tokens("FA", 15, 6), {n: np.asarray(a, dtype=np.float64) for n, a in weights("FA").items()}
    spec = fosovik_spec(read_model_config(FA))
    spec.layers = [replace(spec.layers[0], residual_mult=0.5)]
    spec.order = spec.order[:1]
    model, ops = Decoder(spec), CpuOps()
    model.load({n: torch.tensor(np.asarray(weights("FA")[n])) for n in model.expected_tensors()}, ops, torch.float32)
    cache = PagedCache(model, CacheConfig(page_size=8, max_tokens=64, max_positions=64), torch.float32, "cpu")
    runner, seen = StepRunner(model, cache, ops, torch.float32, "cpu"), []
    runner.layer_probe = lambda i, x: seen.append(x.clone().numpy())
    cache.acquire(1)
    runner.run([StepEntry(1, toks, [])])
    x = W["embed"][toks] * 3.0
    h = fp.squash(x, W, "l0.norm1")
    m = FA["layers"][0]["mixer"]
    want = x + 0.5 * (fp.mamba2(W, "l0.mix.", m, 1e-5, h) + fp.routed_ff(W, "l0.mlp.", 2, h))
    assert np.abs(seen[0] - want).max() <= 2e-5 * np.abs(want).max()
