"""Gedulorn on the CPU: the configuration, the model's structure, the plain functions among themselves, and the engine's host side
(cache slots, a slot that several layers read, windows that give pages back, rows of state, batching, scheduler) over the torch
stand-ins of the kernels."""
import copy
import dataclasses
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import gedulorn_cases as cases
import helpers
from plain import gedulorn_plain as plain

F = torch.float64


@pytest.fixture(scope="module")
def gedulorn_folders(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = cases.make_folder(name, str(tmp_path_factory.mktemp(f"gedulorn_{name.replace('+', '_')}")))
        return made[name]
    return get


def test_configuration_reads_every_size_and_round_trips():
    from vt_transformer_b200.config import ConfigError, config_from_dict
    from vt_transformer_b200.config.gedulorn import GedulornConfig, GedulornRotation
    cfg = config_from_dict(copy.deepcopy(cases.CONFIGS["mix"]))
    assert isinstance(cfg, GedulornConfig) and (cfg.vocab, cfg.width, cfg.embedding_scale, cfg.norm_eps, len(cfg.layers)) == (300, 64, 6.0, 1e-5, 5)
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.scale, m.softcap, m.rot, m.window) == (4, 2, 24, 0.6, 3.0, GedulornRotation(16, 3000.0, 2.5), 17)
    m = cfg.layers[3].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot.dims, m.window, m.kv_from) == (2, 16, 16, 24, 24, 48, 0.25, 16, 45, 1)
    assert cfg.layers[1].mixer.kv_from is None and cfg.layers[4].mixer.softcap is None and cfg.layers[4].mixer.rot.factor == 1.0
    m = cfg.layers[2].mixer
    assert (m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) == (4, 20, 24, 2, 4, 2)
    f = cfg.layers[0].mlp
    assert (f.experts, f.top, f.ff, f.shared_ff) == (5, 2, 20, 36) and cfg.layers[1].mlp.shared_ff is None and cfg.layers[4].mlp is None
    assert config_from_dict(copy.deepcopy(cases.CONFIGS["wide"])).layers[2].mixer.window is None
    for name in cases.CONFIGS:
        one = config_from_dict(cases.config_of(name))
        assert config_from_dict(one.to_dict()) == one
    for spoil, match in ((lambda c: c["layers"][0].__setitem__("type", "other"), "layers\\[0\\].*'other'"),
                         (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "layers\\[1\\].mixer.*'kv_rank'"),
                         (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.*'size'"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 26), "rot.dims"),
                         (lambda c: c["layers"][0]["mixer"].__setitem__("vdim", 16), "vdim"),
                         (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
                         (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 0), "kv_from"),
                         (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 3), "kv_from"),
                         (lambda c: c["layers"][3]["mixer"].__setitem__("kv_rank", 40), "kv_rank"),
                         (lambda c: c["layers"][2]["mixer"].__setitem__("groups", 3), "groups"),
                         (lambda c: c["layers"][2]["mixer"].__setitem__("norm_groups", 3), "norm_groups"),
                         (lambda c: c["layers"][2]["mixer"].pop("conv"), "conv"),
                         (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 6), "top"),
                         (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind 'dense'"),
                         (lambda c: c.pop("norm"), "norm")):
        bad = copy.deepcopy(cases.CONFIGS["mix"])
        spoil(bad)
        with pytest.raises(ConfigError, match=match):
            config_from_dict(bad)


def _build(name):
    from vt_transformer_b200.config import config_from_dict, get_architecture
    from vt_transformer_b200.models.base import DecoderModel
    from vt_transformer_b200.parts import Runtime
    cfg = config_from_dict(cases.config_of(name))
    return DecoderModel(get_architecture(cfg.architecture).model_spec(cfg), Runtime(torch.device("cpu"), torch.float32, None))


def test_what_the_model_reads_and_keeps():
    from vt_transformer_b200.parts import KVCacheSpec, LatentCacheSpec, StateSpec
    model = _build("mix")
    # the slot of layer 1's latent keeps what the wider of its two readers' windows sees
    assert model.cache_slots() == {0: KVCacheSpec(2, 24, 17), 1: LatentCacheSpec(64, 45), 2: StateSpec((4, 24, 20), torch.float32),
                                   3: StateSpec((3, 176), torch.float32), 4: KVCacheSpec(1, 16, 33)}
    assert [(r.cache, r.writes) for r in model.spec.order] == [(0, True), (1, True), ((2, 3), True), (1, False), (4, True)]
    names = model.param_specs()
    assert names["l2.mix.in"].shape == (80 + 176 + 4, 64) and names["l2.mix.conv"].shape == (176, 4) and names["l2.mix.conv.b"].shape == (176,)
    assert names["l0.mix.q.norm"].shape == (24,) and names["l0.mlp.router.b"].shape == (5,) and names["l3.mix.sink"].shape == (2,)
    assert {"embed", "head", "final.norm", "l1.mix.dkv", "l1.mix.dkv.norm", "l2.mix.A_log", "l2.mix.D", "l2.mix.norm", "l0.mlp.shared.up"} <= set(names)
    assert not {"l0.mix.v", "l3.mix.dkv", "l3.mix.dkv.norm", "l4.norm2", "l4.mlp.router", "l1.mlp.shared.up"} & set(names)
    assert model.graph_safe()
    # one tap keeps no inputs; a narrower reader leaves the owner's window as it is
    wide = _build("wide").cache_slots()
    assert wide[4] == StateSpec((2, 70, 18), torch.float32) and len(wide) == 5 and wide[2] == LatentCacheSpec(28, 31)


def test_a_slot_is_as_wide_as_its_widest_reader():
    from vt_transformer_b200.models.base import DecoderModel
    from vt_transformer_b200.parts import KVCacheSpec, LatentCacheSpec, Runtime
    from vt_transformer_b200.parts.base import join_cache_specs
    assert join_cache_specs(LatentCacheSpec(8, 5), LatentCacheSpec(8, 9)) == LatentCacheSpec(8, 9)
    assert join_cache_specs(LatentCacheSpec(8, 5), LatentCacheSpec(8, None)) == LatentCacheSpec(8, None)
    assert join_cache_specs(KVCacheSpec(2, 8, 9, keep_first=3), KVCacheSpec(2, 8, 5, keep_first=4)) == KVCacheSpec(2, 8, 9, keep_first=4)
    for other in (LatentCacheSpec(9, 5), KVCacheSpec(1, 8, 5)):
        with pytest.raises(ValueError):
            join_cache_specs(LatentCacheSpec(8, 5), other)
    spec = _build("mix").spec
    bad = dataclasses.replace(spec, order=spec.order[:3] + (dataclasses.replace(spec.order[3], cache=0),) + spec.order[4:])
    with pytest.raises(ValueError, match="another layout"):
        DecoderModel(bad, Runtime(torch.device("cpu"), torch.float32, None))


def test_rotated_rows_lie_side_by_side():
    from vt_transformer_b200.parts.latent_attention import pairs_side_by_side
    w = torch.arange(12, dtype=torch.float32)[:, None]
    assert pairs_side_by_side(w, [2, 7], 2)[:, 0].tolist() == [0, 1, 2, 4, 3, 5, 6, 7, 9, 8, 10, 11]


def test_plain_functions_agree_with_their_definitions():
    g = torch.Generator().manual_seed(3)
    rand = lambda *s: torch.randn(s, generator=g, dtype=F)
    # the rotation: halves of the first dims, the others pass; twice the factor is half the position
    v = rand(2, 3, 10)
    one = plain.turn_halves(v, torch.tensor([6, 3]), 8, 50.0, 2.0)
    assert torch.allclose(one, plain.turn_halves(v, torch.tensor([3.0, 1.5]), 8, 50.0)) and torch.equal(one[..., 8:], v[..., 8:])
    a = 3 * 50.0 ** (-2 / 8)
    assert torch.allclose(one[0, :, 1], v[0, :, 1] * math.cos(a) - v[0, :, 5] * math.sin(a))
    # the window: itself and the size - 1 tokens before it; the sink takes weight and gives none; the cap bends
    k, vals = rand(6, 1, 4), torch.eye(6, dtype=F)[:, None, :]
    seen = plain.windowed_attention(rand(1, 1, 4), k, vals, torch.tensor([5]), 0.3, 3)[0, 0]
    assert bool((seen[3:] > 0).all()) and float(seen[:3].abs().max()) == 0 and float(seen.sum()) == pytest.approx(1.0)
    q = rand(1, 2, 4)
    zero = plain.windowed_attention(0 * q, k, vals, torch.tensor([5]), 0.3, None, sinks=torch.tensor([0.0, math.log(6.0)], dtype=F))[0]
    assert torch.allclose(zero.sum(-1), torch.tensor([6 / 7, 0.5], dtype=F))
    capped = plain.windowed_attention(1e6 * q, k, vals, torch.tensor([5]), 0.3, None, softcap=2.0)[0]
    assert torch.allclose(capped, torch.softmax(2.0 * torch.sign(torch.einsum("hd,jd->hj", q[0], k[:, 0])), dim=-1))
    # the convolution: the last tap is the present row's, zeros before the start, the same from rows that are kept
    u, w, b = rand(6, 4), rand(4, 3), rand(4)
    out, kept = plain.causal_convolution(u, torch.zeros(2, 4, dtype=F), w, b)
    assert torch.allclose(out[0], plain.silu(b + w[:, 2] * u[0])) and torch.equal(kept, u[4:])
    assert torch.allclose(out[4], plain.silu(b + w[:, 2] * u[4] + w[:, 1] * u[3] + w[:, 0] * u[2]))
    first, kept = plain.causal_convolution(u[:1], torch.zeros(2, 4, dtype=F), w, b)
    rest, kept = plain.causal_convolution(u[1:], kept, w, b)
    assert torch.allclose(torch.cat([first, rest]), out) and torch.equal(kept, u[4:])
    # the recurrence against its closed form: y_t = sum_s C_t . B_s exp(-a sum of the steps behind s) d_s x_s + D x_t
    x, B, C, dt, A, D = rand(5, 2, 3), rand(5, 1, 4), rand(5, 1, 4), plain.softplus(rand(5, 2)), rand(2), rand(2)
    y, S = plain.state_space(x, B, C, dt, A, D, torch.zeros(2, 4, 3, dtype=F), 1)
    for h in range(2):
        ref = D[h] * x[4, h]
        for s in range(5):
            ref = ref + (C[4, 0] @ B[s, 0]) * torch.exp(-torch.exp(A[h]) * dt[s + 1:, h].sum()) * dt[s, h] * x[s, h]
        assert torch.allclose(y[4, h], ref)
    assert torch.allclose(plain.softplus(torch.tensor([-50.0, 0.0, 80.0], dtype=F)), torch.tensor([math.exp(-50.0), math.log(2.0), 80.0], dtype=F))
    # the gate comes before the norm, the norm is over each part by itself
    y, z, w = rand(2, 6), rand(2, 6), rand(6)
    n = plain.gated_group_norm(y, z, w, 2, 1e-9)
    part = (y * plain.silu(z))[:, 3:]
    assert torch.allclose(n[:, 3:], w[3:] * part / part.pow(2).mean(-1, keepdim=True).sqrt())
    # the bias decides the choice; the chosen weights add up to one
    ids, weights = plain.route(0 * rand(3, 8), rand(4, 8), torch.tensor([0.0, 5.0, -1.0, 2.0], dtype=F), 2)
    assert ids.tolist() == [[1, 3]] * 3 and torch.allclose(weights[0], torch.softmax(torch.tensor([5.0, 2.0], dtype=F), 0))


@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_cuts_equal_the_plain_implementation(fake_backend, gedulorn_folders, family):
    cases.replay(gedulorn_folders("mix"), cases.prompts_for("mix"), family, "cpu", "float32")


@pytest.mark.parametrize("name", [n for n in cases.CONFIGS if n not in ("mix", "tensor")])
def test_other_sizes_and_each_mechanism_alone(fake_backend, gedulorn_folders, name):
    prompts = cases.prompts_for(name, lengths=[1, 12, 45])
    for family in ("whole", "portions", "mixed"):
        cases.replay(gedulorn_folders(name), prompts, family, "cpu", "float32", alone=name.endswith("alone"))


def test_tokens_grouped_by_expert_equal_the_plain_implementation(fake_backend, gedulorn_folders, monkeypatch):
    from vt_transformer_b200 import ops
    monkeypatch.setattr(ops, "EXPERTS_GROUPED_MIN_PICKS", 1)
    for name in ("mix", "experts_alone"):
        for family in ("portions", "mixed"):
            cases.replay(gedulorn_folders(name), cases.prompts_for(name, lengths=[1, 9, 40]), family, "cpu", "float32")


def test_every_named_weight_counts(gedulorn_folders, tmp_path):
    """Sinks, the router's bias, the convolution's bias, D, the norms of queries and keys: the plain model without one of them is
    another model by far more than any bound, so a comparison with it shows when the engine leaves one out."""
    for name, ends, value in (("latent_alone", ".sink", -30.0), ("experts_alone", "router.b", 0.0), ("state_alone", "conv.b", 0.0),
                              ("state_alone", ".D", 0.0), ("attention_alone", "k.norm", 1.0), ("state_alone", "mix.norm", 1.0)):
        folder = gedulorn_folders(name)

        def without(t):
            for n in t:
                if n.endswith(ends):
                    t[n] = torch.full_like(t[n], value)
        other = cases.rewritten(folder, str(tmp_path / f"{name}{ends}"), without)
        ids = cases.prompts_for(name)[1]
        ref = helpers.plain_logits(folder, ids)
        assert float((ref - helpers.plain_logits(other, ids)).abs().max()) > 3 * cases.tol("bfloat16", ref, alone=True), (name, ends)


def test_a_window_gives_its_pages_back(fake_backend, gedulorn_folders):
    """A request far longer than every window of the model runs in a pool that could not hold it: each group holds no more pages
    than its widest reader's window and the step's tokens need."""
    from vt_transformer_b200.engine.batch import StepEntry
    folder = gedulorn_folders("mix")
    ids = cases.prompts_for("mix", lengths=[200])[0]
    runner = cases.runner_for(folder, "cpu", "float32", num_pages=5, max_requests=1)
    row, got = runner.admit(), []
    for a in range(0, 200, 8):
        got.append(runner.step([StepEntry(row, ids[a:a + 8], list(range(8)))]).double())
        for g in runner.cache.groups:
            held = g.pool.num_pages - g.pool.free
            assert held <= -(-(g.layout.window + 8) // 16) + 1
    cases.within(torch.cat(got), folder, ids, "float32")
    runner.release(row)
    runner.cache.check()
    assert runner.cache.free_pages() == [5] * len(runner.cache.groups)


def test_a_row_used_again_knows_nothing_of_its_last_request(fake_backend, gedulorn_folders):
    folder = gedulorn_folders("mix")
    runner = cases.runner_for(folder, "cpu", "float32", num_pages=6, max_requests=1)
    for ids in cases.prompts_for("mix", seed=4, lengths=[21, 1, 6, 2]):
        row = runner.admit()
        cases.within(cases.step_all(runner, row, ids, [2, 1, 4]), folder, ids, "float32")
        runner.release(row)


def test_greedy_generation_through_the_entry_point(fake_backend, gedulorn_folders):
    cases.greedy_generation(gedulorn_folders("mix"), "mix", "cpu", "float32", n_new=6)


def test_a_tensor_of_the_wrong_shape_is_refused(fake_backend, gedulorn_folders, tmp_path):
    from vt_transformer_b200.weights import WeightError

    def spoil(t):
        t["l2.mix.conv"] = t["l2.mix.conv"][:, :-1]
    with pytest.raises(WeightError):
        cases.runner_for(cases.rewritten(gedulorn_folders("mix"), str(tmp_path / "bad"), spoil), "cpu", "float32", num_pages=4)


def test_random_weights_mode_of_the_command_line_writes_a_folder_that_loads(tmp_path):
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(cases.CONFIGS["mix"]))
    out = tmp_path / "model"
    res = subprocess.run([sys.executable, "-m", "vt_transformer_b200", "random-weights", "--config", str(cfg), "--out", str(out),
                          "--seed", "5", "--sigma", "0.05"], capture_output=True, text=True, timeout=600,
                         env=dict(os.environ, PYTHONPATH=helpers.ROOT), cwd=helpers.ROOT)
    assert res.returncode == 0, res.stderr
    from vt_transformer_b200.config import config_from_dict, load_config
    from vt_transformer_b200.weights import SafetensorsSource, check_against
    from vt_transformer_b200.weights.random_init import parameter_table
    config = load_config(str(out))
    assert config == config_from_dict(copy.deepcopy(cases.CONFIGS["mix"]))
    check_against(SafetensorsSource(str(out)), parameter_table(config))
