"""Laposun on the CPU: the configuration, the model's structure, the plain functions among themselves, and the engine's
host side (cache slots, windows that give pages back, rows of state, batching, scheduler) over the torch stand-ins of the
kernels."""
import copy
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import helpers
import laposun_cases as cases
from plain import laposun_plain as plain

F = torch.float64


@pytest.fixture(scope="module")
def laposun_folders(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = cases.make_folder(name, str(tmp_path_factory.mktemp(f"laposun_{name.replace('+', '_')}")))
        return made[name]
    return get


def test_configuration_reads_every_size_and_round_trips():
    from vt_transformer_b200.config import ConfigError, config_from_dict
    from vt_transformer_b200.config.laposun import LaposunConfig
    cfg = config_from_dict(copy.deepcopy(cases.CONFIGS["mix"]))
    assert isinstance(cfg, LaposunConfig) and (cfg.vocab, cfg.width, cfg.streams, cfg.taps, len(cfg.layers)) == (300, 64, 2, 3, 4)
    assert (cfg.buckets, cfg.mul_prev, cfg.mul_cur, cfg.norm_eps) == (101, 7, 31, 1e-5)
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot_dims, m.rot_base, m.window) == (3, 24, 16, 40, 40, 48, 0.2, 16, 3000.0, 17)
    f = cfg.layers[0].mlp
    assert (f.experts, f.top, f.scale, f.ff, f.shared_ff) == (5, 2, 2.0, 20, 36)
    assert cfg.layers[1].mlp.ff == 100 and cfg.layers[2].mlp is None and cfg.layers[3].mlp.shared_ff is None
    assert config_from_dict(copy.deepcopy(cases.CONFIGS["wide"])).layers[0].mixer.rot_dims == 4
    for name in cases.CONFIGS:
        one = config_from_dict(cases.config_of(name))
        assert config_from_dict(one.to_dict()) == one
    for spoil, match in ((lambda c: c["layers"][0].__setitem__("type", "other"), "layers\\[0\\].*'other'"),
                         (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "layers\\[1\\].mixer.*'kv_rank'"),
                         (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.*'size'"),
                         (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 18), "rot.dims"),
                         (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 6), "top"),
                         (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "x"), "kind 'x'"),
                         (lambda c: c["canon"].__setitem__("taps", 0), "taps"),
                         (lambda c: c.__setitem__("streams", 17), "streams"),
                         (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
                         (lambda c: c.pop("streams"), "streams")):
        bad = copy.deepcopy(cases.CONFIGS["mix"])
        spoil(bad)
        with pytest.raises(ConfigError, match=match):
            config_from_dict(bad)


def test_what_the_model_reads_and_keeps():
    from vt_transformer_b200.config import config_from_dict, get_architecture
    from vt_transformer_b200.models.base import DecoderModel
    from vt_transformer_b200.parts import LatentCacheSpec, Runtime, StateSpec

    def build(name):
        cfg = config_from_dict(cases.config_of(name))
        return DecoderModel(get_architecture(cfg.architecture).model_spec(cfg), Runtime(torch.device("cpu"), torch.float32, None))
    model = build("mix")
    slots = model.cache_slots()
    rows = StateSpec((2, 64), torch.float32)
    assert slots == {0: StateSpec((1,), torch.int32), 1: rows, 2: rows, 3: LatentCacheSpec(64, 17), 4: rows, 5: rows, 6: LatentCacheSpec(40, 40),
                     7: rows, 8: LatentCacheSpec(56, 16), 9: rows, 10: rows, 11: LatentCacheSpec(64, 33)}
    assert [r.cache for r in model.spec.order] == [(1, 2, 3), (4, 5, 6), (7, 8), (9, 10, 11)]
    names = model.param_specs()
    assert names["bigram"].shape == (102, 64) and names["l0.canon1"].shape == (64, 3) and names["l3.hc2.mix"].shape == (2, 2)
    assert names["l1.hc1.in"].shape == names["l1.hc1.out"].shape == (2,) and names["l2.mix.g"].shape == (4, 64)
    assert names["l0.mlp.shared.sg"].shape == (1, 64) and names["l0.mlp.e4.up"].shape == (20, 64)
    assert {"embed", "embed.norm", "final.norm", "l1.mlp.gate", "l1.norm2", "l0.mix.dkv.norm", "l3.mlp.router"} <= set(names)
    assert not {"l2.norm2", "l2.canon2", "l2.hc2.in", "l0.mlp.e0.gate", "l3.mlp.shared.up", "l3.mlp.shared.sg"} & set(names)
    assert names["head"].optional and model.graph_safe()
    # one tap keeps no rows
    ones = build("ones")
    assert ones.cache_slots() == {0: StateSpec((1,), torch.int32), 1: LatentCacheSpec(24, 12), 2: LatentCacheSpec(12, 25)}
    assert [r.cache for r in ones.spec.order] == [1, 2]


def test_a_model_whose_parts_disagree_about_the_streams_is_refused():
    import dataclasses
    from vt_transformer_b200.config import config_from_dict, get_architecture
    from vt_transformer_b200.models.base import DecoderModel
    from vt_transformer_b200.parts import Runtime
    cfg = config_from_dict(cases.config_of("mix"))
    spec = get_architecture(cfg.architecture).model_spec(cfg)
    rt = Runtime(torch.device("cpu"), torch.float32, None)
    for bad, match in ((dataclasses.replace(spec, streams=3), "streams"), (dataclasses.replace(spec, embedding_cache=None), "slot"),
                       (dataclasses.replace(spec, embedding_cache=2), "slot"),
                       (dataclasses.replace(spec, blocks=spec.blocks[:1] + tuple(dataclasses.replace(b, streams=4) for b in spec.blocks[1:])), "streams")):
        with pytest.raises(ValueError, match=match):
            DecoderModel(bad, rt)


def test_plain_functions_agree_with_their_definitions():
    g = torch.Generator().manual_seed(3)
    rand = lambda *s: torch.randn(s, generator=g, dtype=F)
    # the streams: all change from their old values
    x, mix, w_out, y = rand(3, 2, 5), rand(3, 3), rand(3), rand(2, 5)
    new = plain.write_streams(x, mix, w_out, y)
    for t in range(3):
        assert torch.allclose(new[t], mix[0, t] * x[0] + mix[1, t] * x[1] + mix[2, t] * x[2] + w_out[t] * y)
    assert torch.allclose(plain.read_streams(x, w_out), torch.einsum("s,stw->tw", w_out, x))
    # the convolution: the last tap is the present row's, zeros before the start, the same from rows that are kept
    h, w = rand(6, 4), rand(4, 3)
    out, kept = plain.short_convolution(h, torch.zeros(2, 4, dtype=F), w)
    assert torch.allclose(out[0], h[0] + w[:, 2] * h[0]) and torch.allclose(out[1], h[1] + w[:, 2] * h[1] + w[:, 1] * h[0])
    assert torch.allclose(out[4], h[4] + w[:, 2] * h[4] + w[:, 1] * h[3] + w[:, 0] * h[2]) and torch.equal(kept, h[4:])
    a, kept = plain.short_convolution(h[:1], torch.zeros(2, 4, dtype=F), w)
    b, kept = plain.short_convolution(h[1:5], kept, w)
    c, kept = plain.short_convolution(h[5:], kept, w)
    assert torch.allclose(torch.cat([a, b, c]), out) and torch.equal(kept, h[4:])
    # pairs of tokens
    bg = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert plain.bigram_rows([4, 5, 9], None, bg) == [10, (12 + 35) % 10, (15 + 63) % 10] and plain.bigram_rows([5], 4, bg) == [7]
    # the window: itself and the size - 1 tokens before it
    k, v = rand(6, 1, 4), torch.eye(6, dtype=F)[:, None, :]
    seen = plain.window_attention(rand(1, 1, 4), k, v, torch.tensor([5]), 0.3, 3)[0, 0]
    assert bool((seen[3:] > 0).all()) and float(seen[:3].abs().max()) == 0 and float(seen.sum()) == pytest.approx(1.0)
    # the square of relu; the chosen experts' weights add up to the scale; the gated shared expert
    one = torch.ones((1, 1), dtype=F)
    assert float(plain.expert(3 * one, 2 * one, one)) == 36.0 and float(plain.expert(-3 * one, 2 * one, one)) == 0.0
    ids, weights = plain.route(rand(4, 8), rand(6, 8), 3, 2.5)
    assert torch.allclose(weights.sum(1), torch.full((4,), 2.5, dtype=F)) and bool((weights[:, :-1] >= weights[:, 1:]).all())
    f = {"router": {"top": 1, "scale": 0.0}, "shared": {"ff": 1}}
    w = {"router": one, "e0.up": one, "e0.down": one, "shared.up": one, "shared.down": one, "shared.sg": 0.5 * one}
    assert float(plain.moe_ff(2 * one, w, f)) == pytest.approx(4.0 / (1 + math.exp(-1.0)))


@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_cuts_equal_the_plain_implementation(fake_backend, laposun_folders, family):
    cases.replay(laposun_folders("mix"), cases.prompts_for("mix"), family, "cpu", "float32")


@pytest.mark.parametrize("name", [n for n in cases.CONFIGS if n not in ("mix", "tensor")])
def test_other_sizes_and_each_mechanism_alone(fake_backend, laposun_folders, name):
    prompts = cases.prompts_for(name, lengths=[1, 12, 45])
    for family in ("whole", "portions", "mixed"):
        cases.replay(laposun_folders(name), prompts, family, "cpu", "float32", alone=name.endswith("alone"))


def test_tokens_grouped_by_expert_equal_the_plain_implementation(fake_backend, laposun_folders, monkeypatch):
    from vt_transformer_b200 import ops
    monkeypatch.setattr(ops, "EXPERTS_GROUPED_MIN_PICKS", 1)
    for name in ("mix", "experts_alone"):
        for family in ("portions", "mixed"):
            cases.replay(laposun_folders(name), cases.prompts_for(name, lengths=[1, 9, 40]), family, "cpu", "float32")


def test_a_window_gives_its_pages_back(fake_backend, laposun_folders):
    """A request far longer than every window of the model runs in a pool that could not hold it: each group holds no more
    pages than its window and the step's tokens need."""
    from vt_transformer_b200.engine.batch import StepEntry
    folder = laposun_folders("mix")
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


def test_a_row_used_again_knows_nothing_of_its_last_request(fake_backend, laposun_folders):
    folder = laposun_folders("mix")
    runner = cases.runner_for(folder, "cpu", "float32", num_pages=6, max_requests=1)
    for ids in cases.prompts_for("mix", seed=4, lengths=[21, 1, 6, 2]):
        row = runner.admit()
        cases.within(cases.step_all(runner, row, ids, [2, 1, 4]), folder, ids, "float32")
        runner.release(row)


def test_greedy_generation_through_the_entry_point(fake_backend, laposun_folders):
    cases.greedy_generation(laposun_folders("mix"), "mix", "cpu", "float32", n_new=6)


def test_a_tensor_of_the_wrong_shape_is_refused(fake_backend, laposun_folders, tmp_path):
    from vt_transformer_b200.weights import WeightError

    def spoil(t):
        t["bigram"] = t["bigram"][:-1]
    with pytest.raises(WeightError):
        cases.runner_for(cases.rewritten(laposun_folders("mix"), str(tmp_path / "bad"), spoil), "cpu", "float32", num_pages=4)


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
