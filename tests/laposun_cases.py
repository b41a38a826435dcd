"""Configurations, weights and scenarios of the Laposun tests.  Every scenario runs the engine (``ModelRunner.step`` or
``LLM.generate``) and compares with the plain implementation (tests/plain/laposun_plain.py); each takes the device and
dtype, so the host-side tests run it on the CPU with the stand-in kernels and the GPU tests on cuda:0 with the real ones."""
from __future__ import annotations

import copy
import random
from typing import Dict, List

import numpy as np
import torch

import helpers
from plain import laposun_plain as plain
from sisetar_cases import rewritten, runner_for, step_all  # noqa: F401  (the same helpers serve every design)


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window, mlp=None, dims=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"dims": rot_dim if dims is None else dims, "base": base}, "mask": {"size": window}}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, scale, ff, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff},
            "shared": None if shared is None else {"ff": shared}}


def _model(vocab, width, layers, streams, taps, bigram, eps=1e-5):
    return {"architecture": "Laposun", "vocab": vocab, "width": width, "streams": streams, "canon": {"taps": taps}, "norm": {"eps": eps},
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}


# Configurations that differ from one another in every size and constant: 1 to 7 streams (of which the kernels know 1 to 4
# when they are compiled), 1 to 7 taps (2 to 4 likewise), windows of one token, of less than a page, of whole pages, of one
# token more and less, and longer than the request; values wider and narrower than the plain key part, rotated parts from 4 to 32
# dimensions and one of which only a part turns, latents of a size that is no multiple of 8, one head; experts with top of
# 1 and of all, with and without the shared expert, scores scaled by 1 and by other numbers; inner sizes that are no
# multiple of 8; layers without a feed-forward; one bucket, and factors of 0 and 1 in the pairs' hash.
CONFIGS: Dict[str, dict] = {
    "mix": _model(300, 64, [_lat(3, 24, 16, 40, 40, 48, 0.2, 3000.0, 17, mlp=_moe(5, 2, 2.0, 20, shared=36)),
                            _lat(2, 16, 8, 16, 24, 32, 0.3, 100.0, 40, mlp=_dense(100)),
                            _lat(4, 8, 32, 24, 20, 24, 0.17, 5e4, 16),
                            _lat(3, 24, 16, 40, 40, 48, 0.2, 3000.0, 33, mlp=_moe(6, 1, 0.8, 24))],
                  streams=2, taps=3, bigram=(101, 7, 31)),
    "wide": _model(257, 72, [_lat(1, 40, 8, 24, 12, 20, 0.11, 7.0, 500, mlp=_moe(4, 4, 1.0, 40, shared=24), dims=4),
                             _lat(6, 16, 24, 72, 64, 40, 0.25, 1e6, 31, mlp=_dense(52)),
                             _lat(2, 12, 4, 20, 30, 44, 0.3, 50.0, 1, mlp=_moe(3, 2, 1.7, 12))],
                   streams=7, taps=6, bigram=(37, 1, 0), eps=1e-6),
    "ones": _model(90, 40, [_lat(2, 16, 8, 16, 16, 16, 0.25, 300.0, 12, mlp=_dense(48)),
                            _lat(1, 8, 4, 8, 8, 8, 0.4, 20.0, 25, mlp=_moe(3, 1, 1.0, 8, shared=8))], streams=1, taps=1, bigram=(1, 0, 1)),
    "four": _model(150, 56, [_lat(2, 16, 8, 24, 32, 24, 0.25, 900.0, 64, mlp=_moe(4, 3, 3.0, 16, shared=40)),
                             _lat(3, 8, 12, 16, 16, 32, 0.28, 1e4, 15, mlp=_dense(72))], streams=4, taps=2, bigram=(211, 13, 5)),
    "attention_alone": _model(128, 48, [_lat(4, 16, 8, 24, 24, 32, 0.22, 777.0, 21)], streams=1, taps=1, bigram=(50, 3, 11)),
    "pairs_alone": _model(128, 48, [_lat(1, 8, 4, 8, 8, 8, 0.3, 100.0, 1)], streams=1, taps=1, bigram=(67, 29, 5)),
    "streams_alone": _model(128, 48, [_lat(2, 8, 4, 8, 8, 8, 0.3, 100.0, 9, mlp=_dense(24)), _lat(2, 8, 4, 8, 8, 8, 0.3, 100.0, 9)], streams=3, taps=1,
                            bigram=(9, 2, 1)),
    "convolution_alone": _model(128, 48, [_lat(1, 8, 4, 8, 8, 8, 0.3, 100.0, 1, mlp=_dense(40))], streams=1, taps=5, bigram=(9, 2, 1)),
    "dense_alone": _model(128, 48, [_lat(1, 8, 4, 8, 8, 8, 0.3, 100.0, 1, mlp=_dense(60))], streams=1, taps=1, bigram=(9, 2, 1)),
    "experts_alone": _model(128, 48, [_lat(1, 8, 4, 8, 8, 8, 0.3, 100.0, 1, mlp=_moe(7, 3, 1.4, 28, shared=12))], streams=1, taps=1, bigram=(9, 2, 1)),
    # sizes of the kind a served model has: a latent of 128 with a rotated part of 32 beside it, heads of 64 and 32
    "tensor": _model(200, 128, [_lat(8, 32, 32, 64, 48, 128, 0.12, 1e4, 100, mlp=_moe(3, 3, 1.2, 24, shared=16)),
                                _lat(4, 64, 32, 32, 64, 128, 0.1, 5e5, 130, mlp=_dense(96)),
                                _lat(5, 48, 16, 48, 40, 64, 0.15, 2e4, 64)], streams=3, taps=4, bigram=(401, 211, 3)),
}
SIGMA = {"mix": 0.15, "wide": 0.12, "ones": 0.2, "four": 0.15, "tensor": 0.1}
SEED = {n: 900 + i for i, n in enumerate(CONFIGS)}
LENGTHS = {"mix": [1, 9, 40, 71, 130], "wide": [3, 33, 90, 152], "ones": [1, 2, 30, 66], "four": [1, 17, 64, 110], "tensor": [1, 70, 150, 330, 260]}
LENGTHS.update({n: [1, 25, 66] for n in CONFIGS if n.endswith("alone")})


def every_expert(name: str) -> str:
    """The name of the configuration ``name`` with every router's ``top`` set to its number of experts."""
    return name + "+all"


def for_dtype(name: str, dtype: str) -> str:
    """The configuration that a test of a deep model runs in ``dtype``.  In bfloat16 the rounding of the activations decides
    a router's close call the other way now and then; the token then runs other experts, and through the latents and
    convolutions later positions move by more than rounding explains.  So deep models run in bfloat16 with every expert chosen
    (the weights still come from the scores), and the choice among experts is tested in 32-bit on the same kernels and in
    bfloat16 on the model of one layer, where a close call touches its own position only and is left out."""
    return name if dtype == "float32" else every_expert(name)


def _base(name: str) -> str:
    return name[:-len("+all")] if name.endswith("+all") else name


def config_of(name: str) -> dict:
    cfg = copy.deepcopy(CONFIGS[_base(name)])
    if name.endswith("+all"):
        for layer in cfg["layers"]:
            if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


def settle(name: str):
    """What is done to the random weights: the tables at unit size (the norm behind them brings them there anyway; the pair's
    row then weighs as much as the token's), gates of experts and heads away from one half, and, in the configurations of
    one mechanism, the others taken out: no mixer's result (o = 0), a pair's row of zeros, identical streams."""
    def change(t: Dict[str, torch.Tensor]) -> None:
        for n in list(t):
            if n == "bigram":
                t[n] = (t[n].float() * (0.0 if name.endswith("alone") and name != "pairs_alone" else 1.0)).to(t[n].dtype)
            elif n.endswith(".mix.g") or n.endswith("shared.sg"):
                t[n] = (t[n].float() * 3.0).to(t[n].dtype)
            elif n.endswith(".mix.o") and name in ("pairs_alone", "convolution_alone", "dense_alone", "experts_alone"):
                t[n] = torch.zeros_like(t[n])
            elif ".canon" in n and name.endswith("alone") and name != "convolution_alone":
                t[n] = torch.zeros_like(t[n])
            elif ".hc" in n and name.endswith("alone") and name != "streams_alone":
                t[n] = torch.ones_like(t[n])                      # one stream: u = x, x <- x + y
    return change


def make_folder(name: str, folder: str) -> str:
    from vt_transformer_b200.config import config_from_dict
    from vt_transformer_b200.weights import write_random_model
    made = write_random_model(config_from_dict(config_of(name)), folder + "_raw", seed=SEED[_base(name)], sigma=SIGMA.get(_base(name), 0.2))
    return rewritten(made, folder, settle(_base(name)))


def prompts_for(name: str, seed: int = 0, lengths=None) -> List[List[int]]:
    name = _base(name)
    rng = random.Random(1700 + seed)
    vocab = CONFIGS[name]["vocab"]
    return [[rng.randrange(vocab) for _ in range(n)] for n in (lengths or LENGTHS[name])]


def tol(dtype: str, ref: torch.Tensor, alone: bool = False) -> float:
    """The bound on |logit - plain logit|, as a part of the spread of the model's plain logits.  32-bit differs by
    rounding and the order of sums only; bfloat16 rounds the activations to 8 bits at every part, less in a model of one
    mechanism (``alone``) than in a deep one."""
    spread = max(1.0, float(ref.double().std()))
    return (5e-5 if dtype == "float32" else (0.1 if alone else 0.3)) * spread


def outliers_allowed(dtype: str, n: int) -> int:
    """Positions of ``n`` that may lie beyond the bound: none in 32-bit, one in fifty (at least one) in bfloat16."""
    return 0 if dtype == "float32" else max(1, n // 50)


_close = {}
CLOSE_CALL = 0.03       # a router's margin, as a part of its largest logit, below which bfloat16 rounding may choose otherwise


def close_calls(folder, tokens, dtype) -> set:
    """The positions at which a router of the plain model makes a close call.  Comparisons in bfloat16 leave these
    positions out; in 32-bit every position counts."""
    if dtype == "float32":
        return set()
    key = (folder, tuple(tokens))
    if key not in _close:
        margins = []
        plain.forward(plain.read_config(folder), helpers._plain_weights(folder), list(tokens), margins=margins)
        _close[key] = set(int(i) for m in margins for i in torch.nonzero(m < CLOSE_CALL).flatten())
    return _close[key]


def within(got: torch.Tensor, folder, tokens, dtype, alone: bool = False) -> float:
    """``got`` [T, vocab] against the plain logits of ``tokens``, position by position except at close calls.  Returns the
    worst error as a part of the bound."""
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
    """One way of cutting the requests into steps, with no more pages than the live requests need (so that pages and
    state rows are used again), against the plain implementation.  Returns the worst error as a part of its bound."""
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
    """Scales the weights of the norms of the queries' latents so that a position's attention lies on a few keys, and the
    output projection so that the attention outweighs the embedding: a key that is wrongly seen or wrongly hidden then
    moves the logits far beyond rounding."""
    for n in t:
        if n.endswith("mix.dq.norm") or n.endswith("mix.o"):
            t[n] = (t[n].float() * (4.0 if n.endswith("mix.o") else factor)).to(t[n].dtype)


def with_window(folder, out, window):
    """A copy of a model folder whose attention layers all have that window."""
    def config(c):
        for layer in c["layers"]:
            layer["mixer"]["mask"]["size"] = window
    return rewritten(folder, out, lambda t: None, config=config)


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
