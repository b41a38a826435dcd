"""Laposun on the GPU: the kernels against the plain functions, every mechanism alone and the whole model, through the
engine's step and entry point, against the plain implementation (tests/plain/laposun_plain.py)."""
import math

import pytest
import torch

import helpers
import laposun_cases as cases
from plain import laposun_plain as plain

pytestmark = pytest.mark.gpu
DTYPES = ["bfloat16", "float32"]
DEV = "cuda:0"
F = torch.float64


@pytest.fixture(scope="module")
def laposun_folders(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = cases.make_folder(name, str(tmp_path_factory.mktemp(f"laposun_{name.replace('+', '_')}")))
        return made[name]
    return get


def _logits(folder, tokens):
    return helpers.plain_logits(folder, tokens)


# ----------------------------------------------------------------------------- kernels against the plain functions


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("streams,width", [(1, 48), (2, 200), (3, 4104), (4, 2048), (7, 72), (16, 136)])
def test_streams_kernel(dtype, streams, width):
    """The change of the streams, what is read of them and its norm: without a change, with a tensor and with unadded
    shares, written back or not, over all rows and over some."""
    from vt_transformer_b200 import ops
    g = torch.Generator().manual_seed(width)
    rand = lambda *s: torch.randn(s, generator=g)
    T = 5
    weight, w_in, w_out, mix = 1 + 0.2 * rand(width), rand(streams), rand(streams), rand(streams, streams)
    x, y = rand(T, streams, width), rand(T, width).to(dtype)
    shares = rand(3, T, width)
    rows = torch.tensor([4, 0, 2], dtype=torch.int32)
    dev = lambda t: t.to(DEV)
    eps = 1e-3
    for kind in ("none", "tensor", "shares"):
        full = {"none": None, "tensor": y.double(), "shares": shares.double().sum(0)}[kind]
        want_x = x.double().transpose(0, 1)
        if full is not None:
            want_x = plain.write_streams(want_x, mix.double(), w_out.double(), full)
        want = plain.rms_norm(plain.read_streams(want_x, w_in.double()), weight.double(), eps)
        change = None if full is None else (dev(y) if kind == "tensor" else ops.SplitSum(dev(shares)), dev(mix), dev(w_out))
        for some in (False, True):
            for store in (True, False):
                xd = dev(x)
                out = torch.empty((3 if some else T, width), dtype=dtype, device=DEV)
                ops.streams_norm(xd, dev(w_in), dev(weight), eps, out, change=change, rows=dev(rows) if some else None, store=store)
                ref = want[rows.long()] if some else want
                assert float((out.double().cpu() - ref).abs().max()) <= (2e-5 if dtype == torch.float32 else 3e-2)
                moved = xd.double().cpu().transpose(0, 1)
                before = x.double().transpose(0, 1).clone()
                if store and full is not None:
                    touched = rows.long() if some else torch.arange(T)
                    before[:, touched] = want_x[:, touched]
                assert float((moved - before).abs().max()) <= 2e-5 * max(1.0, float(before.abs().max()))


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("taps,width", [(1, 48), (2, 200), (3, 520), (4, 2056), (4, 7000), (6, 72), (16, 48)])
def test_convolution_carries_its_rows(dtype, taps, width):
    """Norm and convolution over steps of every kind: long portions (several tiles), portions shorter than the taps, single
    tokens (one kernel; two above its width), a sequence that sits a step out.  The rows kept are the unrounded ones."""
    from vt_transformer_b200 import ops
    g = torch.Generator().manual_seed(width + taps)
    rand = lambda *s: torch.randn(s, generator=g)
    weight, conv = 1 + 0.2 * rand(width), 0.5 * rand(taps, width)
    w_in = rand(2)
    tail = torch.zeros((4, max(1, taps - 1), width), device=DEV)
    tail[1] = 7.0                                    # a row that no sequence of the test owns stays as it is
    kept = {r: torch.zeros((taps - 1, width), dtype=F) for r in (0, 2, 3)}
    dev = lambda t: t.to(DEV)
    for lens in ({2: 37, 0: 3}, {2: 1, 0: 1, 3: 1}, {0: 2, 3: 18, 2: 1}, {3: 1}, {2: 2, 0: 16}, {0: 1, 2: 1}):
        ctx = helpers.step_context(list(lens.values()), [0] * len(lens), DEV)
        ctx.rows = torch.tensor(list(lens), dtype=torch.int32, device=DEV)
        x = rand(sum(lens.values()), 2, width)
        out = torch.empty((x.shape[0], width), dtype=dtype, device=DEV)
        ops.streams_norm(dev(x), dev(w_in), dev(weight), 1e-5, out, conv=dev(conv), tail=tail if taps > 1 else None, ctx=ctx)
        h = plain.rms_norm(plain.read_streams(x.double().transpose(0, 1), w_in.double()), weight.double(), 1e-5)
        at = 0
        for row, n in lens.items():
            ref, kept[row] = plain.short_convolution(h[at:at + n], kept[row], conv.double().t())
            assert float((out[at:at + n].double().cpu() - ref).abs().max()) <= (4e-5 if dtype == torch.float32 else 6e-2), (lens, row)
            at += n
        if taps > 1:
            for row in kept:
                assert float((tail[row].double().cpu() - kept[row]).abs().max()) <= 1e-5
    assert taps == 1 or float((tail[1] - 7.0).abs().max()) == 0


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("width,streams,normed", [(48, 3, True), (2120, 1, True), (64, 2, False)])
def test_embedding_by_pairs_of_tokens(dtype, width, streams, normed):
    """Portions and single tokens, the token before from the step or from the state, the last row for a first token, and
    rows of zeros for padding; factors large enough that the hash leaves 32 bits."""
    from vt_transformer_b200 import ops
    g = torch.Generator().manual_seed(width)
    vocab, bg = 90, {"buckets": 33, "mul_prev": 2 ** 31 - 19, "mul_cur": 2 ** 30 + 7}
    table, second = torch.randn((vocab, width), generator=g).to(dtype), torch.randn((34, width), generator=g).to(dtype)
    weight = 1 + 0.2 * torch.randn(width, generator=g) if normed else None
    state = torch.full((3, 1), 55, dtype=torch.int32, device=DEV)
    before, seen = {2: None, 0: None}, {2: 0, 0: 0}
    for lens in ({2: 5, 0: 1}, {2: 1, 0: 1}, {0: 3}, {2: 2, 0: 4}):
        ids = {r: torch.randint(0, vocab, (n,), generator=g).tolist() for r, n in lens.items()}
        ctx = helpers.step_context(list(lens.values()), [seen[r] for r in lens], DEV)
        ctx.rows = torch.tensor(list(lens), dtype=torch.int32, device=DEV)
        flat = sum(ids.values(), [])
        T = len(flat)
        pad = lambda t, v: torch.cat([t, torch.tensor([v], dtype=torch.int32, device=DEV)])
        ctx.token_ids = torch.tensor(flat + [-1], dtype=torch.int32, device=DEV)
        ctx.positions, ctx.token_seq = pad(ctx.positions, 0), pad(ctx.token_seq, -1)
        x = torch.empty((T + 1, streams, width), device=DEV)
        ops.embedding_pair(table.to(DEV), second.to(DEV), ctx, state, x, bg["mul_prev"], bg["mul_cur"],
                           weight=None if weight is None else weight.to(DEV), eps=1e-5)
        at = 0
        for r, n in lens.items():
            rows = plain.bigram_rows(ids[r], before[r], bg)
            ref = table.double()[ids[r]] + second.double()[rows]
            if normed:
                ref = plain.rms_norm(ref, weight.double(), 1e-5)
            for s in range(streams):
                assert float((x[at:at + n, s].double().cpu() - ref).abs().max()) <= 2e-5
            before[r], seen[r], at = ids[r][-1], seen[r] + n, at + n
        assert float(x[T].abs().max()) == 0
        assert int(state[1]) == 55 and all(before[r] is None or int(state[r]) == before[r] for r in before)


@pytest.mark.parametrize("heads,key,v_dim,page,window", [(5, 80, 64, 16, 1), (6, 176, 128, 64, 33), (3, 48, 16, 16, 31), (16, 320, 256, 64, 64),
                                                         (6, 576, 512, 32, 50), (70, 64, 32, 16, 32), (5, 112, 80, 16, 400)])
def test_latent_attention_kernel_under_a_window(heads, key, v_dim, page, window):
    """Rows that all heads share under a window: a sequence that goes on from cached tokens (whose pages before the window
    are gone) beside one that starts; then a step of single tokens.  The values tell the keys apart."""
    from vt_transformer_b200 import ops
    assert ops.backend().attention_latent_supports(key, v_dim)
    g = torch.Generator().manual_seed(heads + key)
    scale = 1.7 / math.sqrt(key)
    lengths = [307 + 70 + 1, 5 + 1]
    rows = [torch.randn((n, key), generator=g).to(torch.bfloat16) for n in lengths]
    n_pages = sum(-(-n // page) for n in lengths) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    pages = torch.full((n_pages, 1, page, key), 3.0, dtype=torch.bfloat16)
    table = torch.full((2, max(-(-n // page) for n in lengths)), -1, dtype=torch.int32)
    for s, r in enumerate(rows):
        for j in range(-(-len(r) // page)):
            table[s, j] = order.pop()
            part = r[j * page:(j + 1) * page]
            pages[table[s, j], 0, :len(part)] = part
    gone = max(0, 307 - window + 1) // page
    table[0, :gone] = -1
    pd, td = pages.to(DEV), table.to(DEV)
    for q_lens, starts in (([70, 5], [307, 0]), ([1, 1], [377, 5]), ([2, 1], [340, 5])):
        T = sum(q_lens)
        q = torch.randn((T, heads, key), generator=g).to(torch.bfloat16)
        ctx = helpers.step_context(q_lens, starts, DEV)
        out = torch.full((T, heads * v_dim), 7.0, dtype=torch.bfloat16, device=DEV)
        ops.attention_latent(q.view(T, -1).to(DEV), 0, out, 0, pd, ctx, td, heads, key, v_dim, scale, window=window)
        at = 0
        for s, (n, start) in enumerate(zip(q_lens, starts)):
            k = rows[s][:start + n].double()
            ref = plain.window_attention(q[at:at + n].double(), k[:, None, :].expand(-1, heads, -1), k[:, None, :v_dim].expand(-1, heads, -1),
                                         torch.arange(start, start + n), scale, window)
            got = out[at:at + n].double().cpu().view(n, heads, v_dim)
            assert float((got - ref).abs().max()) <= 2.5e-2, (q_lens, s)
            at += n


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("tokens", [5, 70])
def test_products_of_the_heads_with_a_gate_a_head(dtype, tokens):
    from vt_transformer_b200 import ops
    g = torch.Generator().manual_seed(tokens)
    heads, inner, outer = 5, 48, 136
    x, m = torch.randn((tokens, heads * inner), generator=g).to(dtype), (torch.randn((heads, inner, outer), generator=g) / 7).to(dtype)
    gate = torch.randn((tokens, 16), generator=g).to(dtype)
    out = torch.empty((tokens, heads * outer), dtype=dtype, device=DEV)
    ops.head_matmul(x.to(DEV), 0, inner, m.to(DEV), out, 0, outer, mode="head_gate", gate=gate.to(DEV), gate_col=8)
    ref = torch.einsum("thi,hio->tho", x.double().view(tokens, heads, inner), m.double()) * torch.sigmoid(gate[:, 8:8 + heads].double())[:, :, None]
    assert float((out.double().cpu().view(tokens, heads, outer) - ref).abs().max()) <= (2e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("m,n,k", [(1, 200, 72), (17, 520, 256), (64, 1000, 136), (200, 384, 512), (600, 640, 64), (1500, 4096, 1536)])
def test_product_with_the_square_of_relu(dtype, m, n, k):
    """Small batches (w as the 128-row operand, with and without cuts of k), tiles of one CTA and of a pair of CTAs."""
    from vt_transformer_b200 import ops
    g = torch.Generator().manual_seed(m)
    x, w = torch.randn((m, k), generator=g).to(dtype).to(DEV), (torch.randn((n, k), generator=g) / math.sqrt(k)).to(dtype).to(DEV)
    out = torch.empty((m, n), dtype=dtype, device=DEV)
    ops.linear_relu_square(x, w, out)
    z = x.double() @ w.double().t()
    ref = z.clamp(min=0.0) ** 2
    assert float(((out.double() - ref).abs() / (1.0 + ref)).max()) <= (1e-5 if dtype == torch.float32 else 8e-3)
    assert float(out[z < -1e-2].abs().max()) == 0


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("experts,top,inter,shared", [(5, 2, 24, 40), (3, 3, 8, 8), (130, 7, 16, 24)])
def test_routing_kernels_with_scaled_scores_and_a_gated_shared_expert(dtype, experts, top, inter, shared):
    """Rows that point along router rows, so that no choice is a close call."""
    from vt_transformer_b200 import ops
    g = torch.Generator().manual_seed(experts)
    T, width = 9, 64
    router, sg = torch.randn((experts, width), generator=g), torch.randn(width, generator=g) / 4
    order = [[(3 * t + 5 * k) % experts for k in range(experts)] for t in range(T)]
    x = torch.stack([sum((top + 2.0 - min(k, top + 1)) * router[order[t][k]] / router[order[t][k]].norm() ** 2 for k in range(min(top + 1, experts)))
                     for t in range(T)]).to(dtype)
    want_ids, want_w = plain.route(x.double(), router.double(), top, 2.2)
    gate = torch.sigmoid(x.double() @ sg.double())
    dev = lambda t: t.to(DEV)
    ids, wts, gates = torch.empty((T, top), dtype=torch.int32, device=DEV), torch.empty((T, top), device=DEV), torch.empty(T, device=DEV)
    ops.route_topk(None, top, ids, wts, x=dev(x), router=dev(router), scale=2.2, shared_gate=dev(sg), gates=gates)
    assert torch.equal(ids.cpu().long().sort(dim=1).values, want_ids.sort(dim=1).values)
    assert float((wts.double().cpu() - want_w).abs().max()) <= 1e-5 and float((gates.double().cpu() - gate).abs().max()) <= 1e-6
    act = torch.rand((T, experts * inter + shared), generator=g).to(dtype)
    ad = dev(act)
    ops.route_experts(None, top, ad, inter, x=dev(x), router=dev(router), scale=2.2, shared_gate=dev(sg))
    dense = torch.zeros((T, experts), dtype=F).scatter(1, want_ids, want_w)
    ref = torch.cat([(act[:, :experts * inter].double().view(T, experts, inter) * dense[:, :, None]).reshape(T, -1),
                     act[:, experts * inter:].double() * gate[:, None]], dim=1)
    assert float((ad.double().cpu() - ref).abs().max()) <= (1e-5 if dtype == torch.float32 else 1.2e-2)
    # the grouped form's last kernel: the picks' rows, and the shared expert's under its gate
    y, sh = torch.randn((T * top, width), generator=g).to(dtype), torch.randn((T, width), generator=g).to(dtype)
    where = torch.randperm(T * top, generator=g).to(torch.int32)
    out = torch.empty((T, width), dtype=dtype, device=DEV)
    ops.combine_picks(dev(y), dev(where), wts, dev(sh), out, gates=gates)
    ref = (wts.double().cpu()[:, :, None] * y.double()[where.long()].view(T, top, width)).sum(1) + gate[:, None] * sh.double()
    assert float((out.double().cpu() - ref).abs().max()) <= (2e-5 if dtype == torch.float32 else 5e-2)


# ----------------------------------------------------------------------------- each mechanism alone


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [n for n in cases.CONFIGS if n.endswith("alone")])
def test_each_mechanism_alone(laposun_folders, name, dtype):
    folder = laposun_folders(name)
    prompts = cases.prompts_for(name, lengths=[1, 12, 45])
    for family in ("whole", "tail", "portions"):
        cases.replay(folder, prompts, family, DEV, dtype, alone=name != "experts_alone")


# ----------------------------------------------------------------------------- the whole model, cut in every way


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "wide", "ones", "four", "tensor"])
@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_cuts_equal_the_plain_implementation(laposun_folders, name, family, dtype):
    page = 64 if name == "tensor" else 16
    cases.replay(laposun_folders(cases.for_dtype(name, dtype)), cases.prompts_for(name), family, DEV, dtype, page_size=page,
                 tail=140 if name == "tensor" else 20, sizes=(40, 3, 64, 2, 150) if name == "tensor" else None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "experts_alone"])
def test_tokens_grouped_by_expert(laposun_folders, monkeypatch, name, dtype):
    """Portions with many picks group their tokens by expert instead of running every expert on every token: forced here
    for every portion, also those in which an expert gets no token."""
    from vt_transformer_b200 import ops
    monkeypatch.setattr(ops, "EXPERTS_GROUPED_MIN_PICKS", 1)
    folder = laposun_folders(cases.for_dtype(name, dtype) if name != "experts_alone" else name)
    for family in ("whole", "portions", "mixed"):
        cases.replay(folder, cases.prompts_for(name), family, DEV, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_two_tokens_and_pages_of_64(laposun_folders, dtype):
    folder = laposun_folders(cases.for_dtype("mix", dtype))
    cases.replay(folder, cases.prompts_for("mix")[1:4], "portions", DEV, dtype, sizes=(2,))
    cases.replay(folder, cases.prompts_for("mix"), "mixed", DEV, dtype, page_size=64)
    cases.replay(folder, cases.prompts_for("mix"), "tail", DEV, dtype, page_size=64, tail=40)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests_equal_each_alone_and_rows_are_used_again(laposun_folders, dtype):
    """Three requests of different lengths stepped together, one of them sitting a step out; then the same rows and
    pages serve other requests.  In 32-bit the logits are those of each request alone, bit for bit."""
    from vt_transformer_b200.engine.batch import StepEntry
    folder = laposun_folders(cases.for_dtype("mix", dtype))
    runner = cases.runner_for(folder, DEV, dtype, num_pages=16, max_requests=3)
    for turn in range(2):
        prompts = cases.prompts_for("mix", seed=turn, lengths=[50, 7, 23])
        alone = []
        for p in prompts:
            row = runner.admit()
            alone.append(cases.step_all(runner, row, p, [len(p)]))
            runner.release(row)
        rows = [runner.admit() for _ in prompts]
        done, got = [0, 0, 0], [[], [], []]
        step = 0
        while any(d < len(p) for d, p in zip(done, prompts)):
            entries, who = [], []
            for i, p in enumerate(prompts):
                if done[i] < len(p) and not (i == 1 and step == 1):
                    k = min([9, 1, 4][(i + step) % 3], len(p) - done[i])
                    entries.append(StepEntry(rows[i], p[done[i]:done[i] + k], list(range(k))))
                    who.append((i, k))
                    done[i] += k
            logits, at = runner.step(entries).double().cpu(), 0
            for i, k in who:
                got[i].append(logits[at:at + k])
                at += k
            step += 1
        runner.check_status()
        for i, p in enumerate(prompts):
            cases.within(torch.cat(got[i]), folder, p, dtype)
            if dtype == "float32":
                assert torch.equal(torch.cat(got[i]), alone[i]), "logits depend on what else is in the batch"
        for r in rows:
            runner.release(r)
        runner.cache.check()


# ----------------------------------------------------------------------------- windows, far keys, page borders, first tokens


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [5, 15, 16, 17, 48, 63, 64, 65])
def test_the_windows_edge_in_prompts_and_in_decoding(laposun_folders, tmp_path, window, dtype):
    """Attention alone, sharpened: the plain logits under windows of one token more and one less differ from the model's far
    beyond the bound at positions past the window, and the engine gives the model's: whole, in portions, decoded alone."""
    sharp = cases.rewritten(laposun_folders("attention_alone"), str(tmp_path / "sharp"), lambda t: cases.sharpen_attention(t, 3.0))
    folder = cases.with_window(sharp, str(tmp_path / "w"), window)
    others = {o: cases.with_window(sharp, str(tmp_path / f"w{o}"), o) for o in (window - 1, window + 1)}
    best = (0.0, None)
    for seed in range(8):                               # the request that shows the edge best, from either side
        ids = cases.prompts_for("attention_alone", seed=seed, lengths=[110])[0]
        shows = []
        for other, near in others.items():
            d = (_logits(near, ids) - _logits(folder, ids)).abs().max(dim=1).values
            assert float(d[:min(window, other)].max()) == 0
            shows.append(float(d[75:].max()))
        if min(shows) > best[0]:
            best = (min(shows), ids)
    ids, ref = best[1], _logits(folder, best[1])
    # (sharpened queries make the scores' rounding in bfloat16 larger: one and a half times the bound of one mechanism)
    bound = cases.tol(dtype, ref, alone=True) * (1.5 if dtype == "bfloat16" else 1.0)
    assert best[0] > 3 * bound
    runner = cases.runner_for(folder, DEV, dtype, num_pages=8, max_requests=1)
    for cuts in ([110], [30, 3, 17, 2, 40, 1, 1], [70] + [1] * 40, [window, 1, 2]):
        row = runner.admit()
        got = cases.step_all(runner, row, ids, cuts)
        runner.release(row)
        assert float((got - ref).abs().max()) <= bound, cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_hundreds_of_tokens_back_and_at_page_borders(laposun_folders, tmp_path, dtype):
    """Attention alone under a window of 388, sharpened so that one key can carry a position's weight: a marked token just
    inside the window, at a page's last place and at the next page's first decides the logits at the asking position, across
    24 pages; whole, in portions, and with the asking tokens decoded one by one."""
    sharp = cases.rewritten(laposun_folders("attention_alone"), str(tmp_path / "sharp"), lambda t: cases.sharpen_attention(t, 4.0))
    folder = cases.with_window(sharp, str(tmp_path / "far"), 388)
    base = cases.prompts_for("attention_alone", seed=2, lengths=[392])[0]
    plain_base = _logits(folder, base)
    # queries four times as long make the scores' rounding in bfloat16 four times as large: twice the bound of a model of
    # one mechanism there (the marked key still moves the logits by more than three times as much)
    bound = cases.tol(dtype, plain_base, alone=True) * (2.0 if dtype == "bfloat16" else 1.0)
    cfg, w = plain.read_config(folder), helpers._plain_weights(folder)
    runner = cases.runner_for(folder, DEV, dtype, num_pages=26, max_requests=1)
    for where in (3, 15, 16, 383):
        best = (0.0, 0, 0)
        for tok in range(0, 128, 2):                    # the token and the asking position that show it best
            ids = list(base)
            ids[where] = tok
            # (position 391 does not see token 3 any more)
            d = (plain.forward(cfg, w, ids)[384:391] - plain_base[384:391]).abs().max(dim=1).values
            best = max(best, (float(d.max()), tok, 384 + int(d.argmax())))
        assert best[0] > 3 * bound, (where, best)
        ids = list(base)
        ids[where] = best[1]
        ref = _logits(folder, ids)
        for cuts in ([len(ids)], [150, 37, 190] + [1] * 15, [380] + [1] * 12):
            row = runner.admit()
            got = cases.step_all(runner, row, ids, cuts)
            runner.release(row)
            assert float((got - ref).abs().max()) <= bound, (where, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["convolution_alone", "pairs_alone", "mix"])
def test_the_first_tokens_and_rows_used_again(laposun_folders, name, dtype):
    """What a request keeps (its last token, the convolutions' rows) must not reach the next request in its row; a stale
    one would show, since the first tokens' logits do depend on what stands before them."""
    folder = laposun_folders(cases.for_dtype(name, dtype))
    a, b = cases.prompts_for(name, lengths=[9, 6])
    runner = cases.runner_for(folder, DEV, dtype, num_pages=2, max_requests=1)
    for ids in (a, b, [b[0]], a):
        for cuts in ([4, 1, 2], [1], [2]):
            row = runner.admit()
            got = cases.step_all(runner, row, ids, cuts)
            runner.release(row)
            ref = _logits(folder, ids)
            assert float((got - ref).abs().max()) <= cases.tol(dtype, ref, alone=name.endswith("alone"))
    ref = _logits(folder, a + b)
    assert float((ref[9:11] - _logits(folder, b)[:2]).abs().max()) > 3 * cases.tol(dtype, ref, alone=name.endswith("alone"))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_beside_a_request_that_joins_and_leaves(laposun_folders, dtype):
    """200 tokens decoded one by one (through the captured graphs of single-token steps, over page borders and past every
    window) beside a second request."""
    from vt_transformer_b200.engine.batch import StepEntry
    folder = laposun_folders(cases.for_dtype("mix", dtype))
    a, b = cases.prompts_for("mix", seed=9, lengths=[201, 40])
    runner = cases.runner_for(folder, DEV, dtype, num_pages=8, max_requests=2)
    ra = runner.admit()
    got_a, got_b, rb = [], [], None
    for i, tok in enumerate(a):
        entries = [StepEntry(ra, [tok], [0])]
        if 30 <= i < 30 + len(b):
            if rb is None:
                rb = runner.admit()
            entries.append(StepEntry(rb, [b[i - 30]], [0]))
        logits = runner.step(entries).double().cpu()
        got_a.append(logits[0])
        if len(entries) == 2:
            got_b.append(logits[1])
            if i - 30 == len(b) - 1:
                runner.release(rb)
    runner.check_status()
    for got, ids in ((got_a, a), (got_b, b)):
        cases.within(torch.stack(got), folder, ids, dtype)
    assert runner._graphs, "single-token steps did not run as captured graphs"


# ----------------------------------------------------------------------------- the entry point


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "four"])
def test_greedy_generation_through_the_entry_point(laposun_folders, name, dtype):
    cases.greedy_generation(laposun_folders(cases.for_dtype(name, dtype)), name, DEV, dtype)


def test_trace_replay_command(laposun_folders, tmp_path):
    folder = laposun_folders("mix")
    prompts = cases.prompts_for("mix")
    trace = helpers.trace_mixed(prompts, max_live=4, seed=2)
    got = helpers.run_trace_cli(folder, trace, "float32", str(tmp_path / "out"), helpers.tokens_needed(trace, 64))
    cases.compare(folder, prompts, trace, got, "float32")


def test_generate_from_the_command_line_greedy(laposun_folders):
    import os
    import subprocess
    import sys
    folder = laposun_folders("four")
    prompts = cases.prompts_for("four")[:2]
    base = [sys.executable, "-m", "vt_transformer_b200", "generate", "--model", folder, "--dtype", "float32", "--max-tokens", "6",
            "--ignore-eos", "--num-pages", "16", "--max-seq-len", "128", "--page-size", "16", "--temperature", "0"]
    for p in prompts:
        base += ["--prompt-ids", ",".join(str(t) for t in p)]
    res = subprocess.run(base, capture_output=True, text=True, timeout=600, env=dict(os.environ, PYTHONPATH=helpers.ROOT), cwd=helpers.ROOT)
    assert res.returncode == 0, res.stderr[-3000:]
    lines = [[int(t) for t in l.split()] for l in res.stdout.splitlines() if l.strip()]
    assert len(lines) == 2 and all(len(l) == 6 for l in lines)
    for p, o in zip(prompts, lines):
        ref = _logits(folder, list(p) + o)
        for i, tok in enumerate(o):
            row = ref[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 2 * cases.tol("float32", ref)
