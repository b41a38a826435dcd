"""Configurations, weights and scenarios of the Gedulorn tests.  Every scenario runs the engine (``ModelRunner.step`` or
``LLM.generate``) and compares with the plain implementation (tests/plain/gedulorn_plain.py); each takes the device and dtype, so
the host-side tests run it on the CPU with the stand-in kernels and the GPU tests on cuda:0 with the real ones."""
from __future__ import annotations

import copy
import random
from typing import Dict, List

import numpy as np
import torch

import helpers
from plain import gedulorn_plain as plain
from sisetar_cases import rewritten, runner_for, step_all  # noqa: F401  (the same helpers serve every design)


def _att(heads, kv_heads, dim, rot, base, scale, window, softcap=None, factor=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap,
                      "rot": {"dims": rot, "base": base, **({} if factor is None else {"scaling": {"factor": factor}})},
                      "mask": None if window is None else {"size": window}}}


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window, mlp=None, kv_from=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"dims": rot_dim, "base": base}, "mask": None if window is None else {"size": window},
                      **({} if kv_from is None else {"kv_from": kv_from})}}


def _ssm(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def _moe(experts, top, ff, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": None if shared is None else {"ff": shared}}


def _model(vocab, width, layers, scale, eps=1e-5):
    return {"architecture": "Gedulorn", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


# Configurations that differ from one another in every size and constant: heads as many as key/value heads and several a
# key/value head, one head; rotations of the whole head, of a part and of none, with and without a factor; caps that bend every
# score, that bend few, and none; windows of one token, of less than a page, of whole pages, of a token more and less, longer than
# the request, and none; layers over another layer's latent with the same window, a wider and a narrower one, over a layer further back and two over
# one layer; latents of a size that is no multiple of 8; states smaller and larger than a value, of sizes that are no multiple of 4
# or 16, values wider than the 64 columns of a CTA; one group and a group a head; one to six taps; one norm group and several; top of 1
# and of all, with and without the shared expert, inner sizes that are no multiple of 8, layers without a feed-forward.
CONFIGS: Dict[str, dict] = {
    "mix": _model(300, 64, [_att(4, 2, 24, 16, 3000.0, 0.6, 17, softcap=3.0, factor=2.5, mlp=_moe(5, 2, 20, shared=36)),
                            _lat(3, 24, 16, 40, 40, 48, 0.2, 900.0, 21, mlp=_moe(4, 3, 24)),
                            _ssm(4, 20, 24, 2, 4, 2, mlp=_moe(6, 1, 16, shared=24)),
                            _lat(2, 16, 16, 24, 24, 48, 0.25, 900.0, 45, kv_from=1, mlp=_moe(3, 2, 12, shared=20)),
                            _att(3, 1, 16, 16, 50.0, 0.4, 33)], scale=6.0),
    "wide": _model(257, 72, [_ssm(3, 66, 20, 1, 6, 1, mlp=_moe(4, 4, 40, shared=24)), _lat(1, 40, 8, 24, 12, 20, 0.11, 7.0, 31),
                             _att(2, 2, 40, 20, 1e6, 0.3, None, softcap=20.0, mlp=_moe(3, 2, 12)), _ssm(2, 18, 70, 2, 1, 4),
                             _lat(6, 16, 8, 72, 64, 20, 0.25, 7.0, 9, kv_from=1, mlp=_moe(7, 3, 28, shared=12)),
                             _lat(2, 12, 8, 16, 30, 20, 0.3, 7.0, 31, kv_from=1)], scale=8.0, eps=1e-6),
    "ones": _model(90, 40, [_ssm(1, 8, 8, 1, 2, 1, mlp=_moe(3, 1, 8, shared=8)), _att(1, 1, 8, 0, 20.0, 0.5, 12, mlp=_moe(1, 1, 16)),
                            _lat(1, 8, 4, 8, 8, 8, 0.4, 20.0, 25)], scale=5.0),
    "attention_alone": _model(128, 48, [_att(4, 2, 16, 8, 777.0, 0.5, 21, softcap=6.0, factor=3.0)], scale=5.0),
    "latent_alone": _model(128, 48, [_lat(4, 16, 8, 24, 24, 32, 0.22, 777.0, 21)], scale=5.0),
    "shared_latent_alone": _model(128, 48, [_lat(2, 16, 8, 24, 24, 32, 0.22, 777.0, 5), _lat(4, 8, 8, 16, 32, 32, 0.3, 777.0, 21, kv_from=0)], scale=5.0),
    "state_alone": _model(128, 48, [_ssm(4, 12, 20, 2, 3, 2)], scale=5.0),
    "experts_alone": _model(128, 48, [_att(1, 1, 8, 8, 100.0, 0.3, 1, mlp=_moe(7, 3, 28, shared=12))], scale=5.0),
    # sizes of the kind a served model has: heads of 64 and 128, a latent of 128 beside a rotated part of 32, states of 128 and 64
    "tensor": _model(200, 128, [_att(8, 2, 64, 32, 1e5, 0.2, 100, softcap=8.0, factor=4.0, mlp=_moe(3, 3, 24, shared=16)),
                                _ssm(6, 64, 128, 2, 4, 2, mlp=_moe(3, 3, 24, shared=16)),
                                _lat(8, 32, 32, 64, 48, 128, 0.12, 1e4, 100),
                                _ssm(4, 32, 64, 1, 3, 1, mlp=_moe(2, 2, 40)),
                                _lat(4, 64, 32, 32, 64, 128, 0.1, 1e4, 130, kv_from=2),
                                _att(3, 3, 128, 128, 5e5, 0.1, 64)], scale=9.0),
}
SIGMA = {"mix": 0.15, "wide": 0.12, "ones": 0.2, "tensor": 0.1}
SEED = {n: 400 + i for i, n in enumerate(CONFIGS)}
LENGTHS = {"mix": [1, 9, 40, 71, 130], "wide": [3, 33, 90, 152], "ones": [1, 2, 30, 66], "tensor": [1, 70, 150, 330, 260]}
LENGTHS.update({n: [1, 25, 66] for n in CONFIGS if n.endswith("alone")})


def every_expert(name: str) -> str:
    """The name of the configuration ``name`` with every router's ``top`` set to its number of experts."""
    return name + "+all"


def for_dtype(name: str, dtype: str) -> str:
    """The configuration that a test of a deep model runs in ``dtype``.  In bfloat16 the rounding of the activations decides a
    router's close call the other way now and then; the token then runs other experts, and through keys and states later
    positions move by more than rounding explains.  So deep models run in bfloat16 with every expert chosen (the weights still
    come from the scores), and the choice among experts is tested in 32-bit on the same kernels and in bfloat16 on the model of
    one layer, where a close call touches its own position only and is left out."""
    return name if dtype == "float32" else every_expert(name)


def _base(name: str) -> str:
    return name[:-len("+all")] if name.endswith("+all") else name


def config_of(name: str) -> dict:
    cfg = copy.deepcopy(CONFIGS[_base(name)])
    if name.endswith("+all"):
        for layer in cfg["layers"]:
            if layer["mlp"] is not None:
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


def settle(name: str):
    """What is done to the random weights: sinks, the router's bias, the convolution's bias and the step sizes' bias of a size that
    counts; norms of queries and keys away from one (a value that were taken after the norm would show); and, in the model of the
    experts alone, no mixer's result (o = 0)."""
    def change(t: Dict[str, torch.Tensor]) -> None:
        for n in list(t):
            if n.endswith(".sink"):
                t[n] = (t[n].float() * 8.0 + 1.0).to(t[n].dtype)
            elif n.endswith("router.b") or n.endswith("conv.b"):
                t[n] = (t[n].float() * 4.0).to(t[n].dtype)
            elif n.endswith("dt_bias"):
                t[n] = (t[n].float() * 4.0 - 1.0).to(t[n].dtype)
            elif n.endswith("mix.q.norm") or n.endswith("mix.k.norm"):
                t[n] = (1.0 + 3.0 * (t[n].float() - 1.0)).to(t[n].dtype)
            elif n.endswith(".mix.o") and name == "experts_alone":
                t[n] = torch.zeros_like(t[n])
    return change


def make_folder(name: str, folder: str) -> str:
    from vt_transformer_b200.config import config_from_dict
    from vt_transformer_b200.weights import write_random_model
    made = write_random_model(config_from_dict(config_of(name)), folder + "_raw", seed=SEED[_base(name)], sigma=SIGMA.get(_base(name), 0.2))
    return rewritten(made, folder, settle(_base(name)))


def prompts_for(name: str, seed: int = 0, lengths=None) -> List[List[int]]:
    name = _base(name)
    rng = random.Random(2900 + seed)
    vocab = CONFIGS[name]["vocab"]
    return [[rng.randrange(vocab) for _ in range(n)] for n in (lengths or LENGTHS[name])]


def tol(dtype: str, ref: torch.Tensor, alone: bool = False) -> float:
    """The bound on |logit - plain logit|, as a part of the spread of the model's plain logits.  32-bit differs by rounding and the
    order of sums only; bfloat16 rounds the activations to 8 bits at every part, less in a model of one mechanism (``alone``) than
    in a deep one."""
    spread = max(1.0, float(ref.double().std()))
    return (1e-4 if dtype == "float32" else (0.1 if alone else 0.3)) * spread


def outliers_allowed(dtype: str, n: int) -> int:
    """Positions of ``n`` that may lie beyond the bound: none in 32-bit, one in fifty (at least one) in bfloat16."""
    return 0 if dtype == "float32" else max(1, n // 50)


_close = {}
CLOSE_CALL = 0.03       # a router's margin, as a part of its largest logit, below which bfloat16 rounding may choose otherwise


def close_calls(folder, tokens, dtype) -> set:
    """The positions at which a router of the plain model makes a close call.  Comparisons in bfloat16 leave these positions
    out; in 32-bit every position counts."""
    if dtype == "float32":
        return set()
    key = (folder, tuple(tokens))
    if key not in _close:
        margins = []
        plain.forward(plain.read_config(folder), helpers._plain_weights(folder), list(tokens), margins=margins)
        _close[key] = set(int(i) for m in margins for i in torch.nonzero(m < CLOSE_CALL).flatten())
    return _close[key]


def within(got: torch.Tensor, folder, tokens, dtype, alone: bool = False) -> float:
    """``got`` [T, vocab] against the plain logits of ``tokens``, position by position except at close calls.  Returns the worst
    error as a part of the bound."""
    ref = helpers.plain_logits(folder, tokens)
    keep = [i for i in range(len(tokens)) if i not in close_calls(folder, tokens, dtype)]
    assert bool(torch.isfinite(got).all()) and 3 * len(keep) >= len(tokens)
    d = (got[keep].double() - ref[keep]).abs().max(dim=1).values
    over = int((d > tol(dtype, ref, alone)).sum())
    assert over <= (0 if alone else outliers_allowed(dtype, len(keep))), (over, float(d.max()), tol(dtype, ref, alone))
    return float(d.max()) / tol(dtype, ref, alone)


def compare(folder, prompts, trace, got, dtype, alone: bool = False) -> float:
    worst, counted, total, over = 0.0, 0, 0, []
    for n in sorted(trace.expect):
        exp = trace.expect[n]
        assert got[n].shape[0] == len(exp), f"step {n}: {got[n].shape[0]} rows, {len(exp)} wanted"
        for i, (r, pos) in enumerate(exp):
            ref = helpers.plain_logits(folder, prompts[r])
            total += 1
            if pos in close_calls(folder, prompts[r], dtype):
                assert np.isfinite(got[n][i]).all()
                continue
            counted += 1
            d = float(np.abs(got[n][i].astype(np.float64) - ref[pos].numpy()).max())
            bound = tol(dtype, ref, alone)
            assert np.isfinite(d)
            worst = max(worst, d / bound)
            if d > bound:
                over.append(f"step {n}, request {r} (length {len(prompts[r])}), position {pos}: |dlogit| {d:.3e} > {bound:.1e} "
                            f"(entries {[(e['id'], len(e['tokens'])) for e in trace.steps[n]['entries']]})")
    assert len(over) <= (0 if alone else outliers_allowed(dtype, counted)), over
    assert 3 * counted >= total, f"only {counted} of {total} positions are free of a router's close call: the test compares too little"
    return worst


def replay(folder, prompts, family, device, dtype, page_size=16, sizes=None, tail=20, alone: bool = False) -> float:
    """One way of cutting the requests into steps, with no more pages than the live requests need (so that pages and state rows
    are used again), against the plain implementation.  Returns the worst error as a part of its bound."""
    make = {"whole": helpers.trace_whole, "tail": lambda p: helpers.trace_tail(p, tail=tail),
            "portions": (lambda p: helpers.trace_portions(p, sizes=sizes)) if sizes else helpers.trace_portions,
            "mixed": lambda p: helpers.trace_mixed(p, max_live=3, seed=5)}[family]
    trace = make(prompts)
    pages = max(1, helpers.tokens_needed(trace, round_to=page_size) // page_size)
    runner = runner_for(folder, device, dtype, num_pages=pages, max_requests=3 if family == "mixed" else 1, page_size=page_size)
    got = helpers.run_trace_inproc(runner, trace)
    worst = compare(folder, prompts, trace, got, dtype, alone)
    assert runner.cache.free_pages() == [g.pool.num_pages for g in runner.cache.groups]
    assert runner.cache.free_rows == runner.cache.max_requests
    runner.cache.check()
    return worst


def sharpen_attention(t: Dict[str, torch.Tensor], factor: float = 4.0) -> None:
    """Scales the weights of the queries' norms so that a position's attention lies on a few keys, and takes the sinks back so
    that they leave the keys their weight: a key that is wrongly seen or wrongly hidden then moves the logits far beyond rounding."""
    for n in t:
        if n.endswith("mix.dq.norm") or n.endswith("mix.q.norm"):
            t[n] = (t[n].float() * factor).to(t[n].dtype)
        elif n.endswith(".sink"):
            t[n] = torch.full_like(t[n], -2.0)
        elif n.endswith("norm1"):
            t[n] = (t[n].float() * 2.0).to(t[n].dtype)


def with_window(folder, out, window, layer=None):
    """A copy of a model folder whose attention layers (or the layer of that number) have that window, and no cap on scores."""
    def config(c):
        for i, entry in enumerate(c["layers"]):
            if "mask" in entry["mixer"] and (layer is None or i == layer):
                entry["mixer"]["mask"] = {"size": window}
            if "softcap" in entry["mixer"]:
                entry["mixer"]["softcap"] = None
    return rewritten(folder, out, lambda t: None, config=config)


def remember(t: Dict[str, torch.Tensor]) -> None:
    """State-space heads that hardly forget and take small steps, read strongly: what a token hundreds back put into the state
    still decides the logits."""
    for n in t:
        if n.endswith("A_log"):
            t[n] = torch.full_like(t[n], -7.0)
        elif n.endswith("dt_bias"):
            t[n] = torch.full_like(t[n], -1.5)
        elif n.endswith("norm1"):
            t[n] = (t[n].float() * 3.0).to(t[n].dtype)


def greedy_generation(folder, name, device, dtype, n_new=12):
    """Greedy generation through the entry point and its scheduler (portions of prompts beside decoding requests)."""
    from vt_transformer_b200 import LLM, SamplingParams
    prompts = prompts_for(name)[1:4]
    llm = LLM(folder, dtype=dtype, device=device, max_running_reqs=3, num_pages=24, max_seq_len=192, page_size=16,
              max_extend_tokens=40, chunk_size=24)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n_new, ignore_eos=True))
    cfg, w = plain.read_config(folder), helpers._plain_weights(folder)
    for p, o in zip(prompts, outs):
        assert len(o) == n_new
        ref = plain.forward(cfg, w, list(p) + o)
        close = close_calls(folder, list(p) + o, dtype)
        for i, tok in enumerate(o):
            if len(p) - 1 + i in close:
                continue
            row = ref[len(p) - 1 + i]
            # the token is the plain argmax, or (two logits closer than the rounding) its plain logit is within the bound
            assert float(row.max() - row[tok]) <= 2 * tol(dtype, ref), (len(p), i, tok)
    llm.runner.cache.check()
    assert llm.stats["free_pages"] == [24] * len(llm.runner.cache.groups)
    return outs
