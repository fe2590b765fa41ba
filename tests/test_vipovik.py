"""Vipovik models through the engine against the plain implementation (GPU): whole prompts, portions down to two tokens,
token-by-token decoding through captured graphs, batches of unequal requests beside each alone, pages and request slots
used again, tokens just inside and just outside windows and among the first ones, a state that has to last, long decoding,
odd sizes, greedy generation through the scheduler, and trace replay."""
import copy

import numpy as np
import pytest
import torch

from vipovik_helpers import (MIXED, ODD, ONE_LAYER, REAL, WIDE, assert_close, config, layer, left, make_engine, make_weights,
                             mixed_schedule, plain, plain_all, rounding_moves, run_cut, tokens_of, unrouted)

pytestmark = pytest.mark.gpu


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["attention", "time_mixing", "side_by_side", "loop", "routed", "mixed", "odd",
                                  "mixed_without_experts", "odd_without_experts"])
def test_whole_prompt_portions_and_single_tokens(name, dtype):
    """A whole prompt; portions of several sizes down to two tokens that end inside pages; token by token from the first
    token on (decode steps, which replay captured graphs): all against the plain implementation.  Small models hold one
    mechanism each."""
    cfgd = {"mixed": MIXED, "odd": ODD, "mixed_without_experts": unrouted(MIXED),
            "odd_without_experts": unrouted(ODD)}.get(name) or ONE_LAYER[name]
    w = make_weights(cfgd, 7)
    toks = tokens_of(cfgd, 75, 3)
    ref, _, close = plain_all(cfgd, w, toks)
    moves = rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None
    eng = make_engine(cfgd, w, dtype)
    for sizes in ([75], [13, 2, 9, 3, 16, 2, 30], [40] + [1] * 35, [2], [1]):
        assert_close(run_cut(eng, toks, sizes), ref, dtype, (name, sizes), close, moves=moves)


def test_the_residual_stream_after_every_layer_run():
    """32-bit, the stream as every block of the running model leaves it, in every pass, against the plain one."""
    from cbis_b200.parts.blocks import ScaledPreNormBlock, _add_pending
    w = make_weights(MIXED, 21)
    toks = tokens_of(MIXED, 40, 9)
    _, ref, _ = plain_all(MIXED, w, toks)
    eng = make_engine(MIXED, w, "float32")
    seen, run = [], ScaledPreNormBlock.forward

    def keep(self, ctx, x, pending, cache, state):
        d = run(self, ctx, x, pending, cache, state)
        after = x.clone()
        if d is not None:
            _add_pending(ctx, after, d)
        seen.append(after.double().cpu())
        return d
    ScaledPreNormBlock.forward = keep
    try:
        run_cut(eng, toks, [40])
    finally:
        ScaledPreNormBlock.forward = run
    assert len(seen) == len(ref) == 11
    for n, (got, want) in enumerate(zip(seen, ref)):
        assert (got - want).abs().max() < 1e-4 * max(1.0, want.abs().max().item()), n


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["wide", "wide_without_experts"])
def test_sizes_of_the_tiled_kernels(name, dtype):
    cfgd = WIDE if name == "wide" else unrouted(WIDE)
    w = make_weights(cfgd, 17, std=0.15)
    toks = tokens_of(cfgd, 220, 5)
    ref, _, close = plain_all(cfgd, w, toks)
    moves = rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None
    eng = make_engine(cfgd, w, dtype, page_size=16, num_pages=40, max_batched_tokens=256)
    for sizes in ([220], [100, 3, 64, 2, 51], [170] + [1] * 50):
        assert_close(run_cut(eng, toks, sizes), ref, dtype, sizes, close, tol32=1e-3, moves=moves)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_as_wide_as_a_small_real_model(dtype):
    """Width 512, a prompt of 300 tokens: the products run on the TMA + tcgen05 kernels, the experts in tiles over rows
    sorted by expert, the recurrence in pieces, attention of head size 64 on the tensor-core kernels."""
    cfgd = REAL
    w = make_weights(cfgd, 19, std=0.12)
    toks = tokens_of(cfgd, 300, 5)
    ref, _, close = plain_all(cfgd, w, toks)
    moves = rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None
    eng = make_engine(cfgd, w, dtype, page_size=16, num_pages=40, max_batched_tokens=512)
    for sizes in ([300], [150, 2, 148], [270] + [1] * 30):
        assert_close(run_cut(eng, toks, sizes), ref, dtype, sizes, close, tol32=2e-3, moves=moves)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "mixed_without_experts"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(name, dtype):
    """Six requests through three slots and a pool smaller than the requests together: portions of some beside single
    tokens of others; every logit equals the request's alone.  Freed pages are filled with NaN before they are used
    again (those behind windows too, while the first tokens' pages stay)."""
    cfgd = {"mixed": MIXED, "odd": ODD}.get(name) or unrouted(MIXED)
    w = make_weights(cfgd, 9)
    lens = {"a": 70, "b": 33, "c": 58, "d": 2, "e": 47, "f": 64}
    seqs = {r: tokens_of(cfgd, n, 40 + i) for i, (r, n) in enumerate(lens.items())}
    plan = {"a": [30, 2, 1, 1, 1, 1, 1, 33], "b": [2, 20, 1, 1, 1, 8], "c": [50, 1, 1, 2, 1, 1, 1, 1], "d": [2],
            "e": [3, 1, 1, 1, 41], "f": [17, 40, 1, 1, 1, 1, 1, 1, 1]}
    assert all(sum(plan[r]) == lens[r] for r in lens)
    eng = make_engine(cfgd, w, dtype, num_pages=26, max_num_seqs=3, poison_freed_pages=True)
    got = mixed_schedule(eng, seqs, plan, list(lens))
    assert eng.pages_poisoned > 10
    for r in lens:
        ref, _, close = plain_all(cfgd, w, seqs[r])
        assert_close(got[r], ref, dtype, r, close, moves=rounding_moves(cfgd, w, seqs[r]) if dtype == "bfloat16" else None)
        if dtype == "float32" or name == "mixed_without_experts":       # beside the request's own run, alone and whole
            alone = run_cut(eng, seqs[r], [lens[r]])
            assert (got[r] - alone).abs().max() < (2e-4 if dtype == "float32" else 0.06 * alone.abs().max()), r


# ---- weights made so that a fault shows ------------------------------------------------------------------------
def _stand_out(t):
    """Token 5's key stands out for every query of the layer: the token's row of the table is one large entry, which the
    last entry of every key head picks up; a query's last entry comes from an entry that every token's row has."""
    t["embed"] *= 0.3
    t["embed"][:, 0] = 0.0
    t["embed"][:, 1] = 2.0
    t["embed"][5, 0] = 8.0
    t["l0.norm1"].fill_(1.0)
    for n, c in (("q", 1), ("k", 0)):
        m = t["l0.mix.left." + n]
        m *= 0.2
        m[:, :2] = 0.0
        m[15::16, c] = 2.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window, keep", [(40, 9), (24, 1), (7, 64), (None, 0), (33, 0)])
def test_one_token_inside_and_outside_of_the_window_and_among_the_first(window, keep, dtype):
    """A one-layer model in which one token's key outweighs all others: it decides every row that sees it, the last one
    inside the window among them, and no row that does not.  The last kept token and the first one not kept, tokens at pages'
    borders and inside a page.  Whole, in portions and token by token."""
    for place in sorted({0, max(keep - 1, 0), keep, 8, 63, 41}):
        cfgd = config(64, 80, [layer(left(4, 2, 16, 16, 1.5, window, keep, 20.0, {"base": 100.0, "dims": 12}), 1, 8, 4, None, 1.0, 0.0)])
        w = make_weights(cfgd, 31, tweak=_stand_out)
        toks = [t if t != 5 else 6 for t in tokens_of(cfgd, 160, 12)]
        toks[place] = 5
        ref = plain(cfgd, w, toks)
        other = plain(cfgd, w, [t if i != place else 7 for i, t in enumerate(toks)])
        diff = (ref - other).abs().max(1).values
        sees = [i for i in range(place + 1, 160) if window is None or i - place < window or place < keep]
        blind = [i for i in range(place + 1, 160) if i not in sees]
        assert diff[sees].min() > 0.1 and (not blind or diff[blind].max() < 1e-9), place
        eng = make_engine(cfgd, w, dtype, poison_freed_pages=True)
        for sizes in ([160], [39, 2, 40, 38, 2, 39], [8, 2, 6] + [1] * 80 + [64]):
            got = run_cut(eng, toks, sizes)
            assert_close(got, ref, dtype, (place, sizes))
            assert (got - ref).abs().max() < 0.3 * diff[sees].min() or dtype == "float32"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_that_has_to_last(dtype):
    """Time mixing whose decays are almost one: a token far back still shows in every later row, across portions, decode
    steps and passes; a lost or doubled state would too."""
    def slow(t):
        for n in t:
            if n.endswith(".w0"):
                t[n].fill_(-9.0)
            if n.endswith(".w2"):
                t[n].mul_(0.02)
    cfgd = config(64, 80, [layer(left(1, 1, 8, 8, 0.4, 2), 2, 16, 12, None, 0.0, 1.5)], loop=(0, 1, 2))
    w = make_weights(cfgd, 33, tweak=slow)
    toks = tokens_of(cfgd, 240, 14)
    ref = plain(cfgd, w, toks)
    other = plain(cfgd, w, [t if i != 3 else (t + 1) % 80 for i, t in enumerate(toks)])
    assert (ref - other).abs().max(1).values[-40:].max() > 0.05
    eng = make_engine(cfgd, w, dtype)
    moves = rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None
    for sizes in ([240], [2, 2, 50, 130, 56], [20] + [1] * 220):
        assert_close(run_cut(eng, toks, sizes), ref, dtype, sizes, moves=moves)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    cfgd = MIXED if dtype == "float32" else unrouted(MIXED)
    w = make_weights(cfgd, 11)
    toks = tokens_of(cfgd, 300, 4)
    ref, _, close = plain_all(cfgd, w, toks)
    moves = rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None
    eng = make_engine(cfgd, w, dtype)
    assert_close(run_cut(eng, toks, [20] + [1] * 280), ref, dtype, "decode", close, tol32=5e-4, moves=moves)


def test_two_scales_and_a_zero():
    """Constants of the two mixers that are equal, unlike, negative and zero (a mixer times zero still keeps its cache and
    state), and one: the product then adds into the stream itself (32-bit and bfloat16)."""
    for ls, rs in ((1.0, 1.0), (0.6, 0.6), (2.0, -0.5), (0.0, 0.9), (1.3, 0.0), (1.0, 0.25), (0.0, 0.0)):
        cfgd = config(64, 80, [layer(left(2, 1, 16, 16, 0.4, 9, 2), 2, 16, 6, None, ls, rs), layer(left(2, 2, 8, 8, 0.4), 1, 8, 6, None, rs, ls)])
        w = make_weights(cfgd, 5)
        toks = tokens_of(cfgd, 40, 6)
        ref = plain(cfgd, w, toks)
        for dtype in ("float32", "bfloat16"):
            moves = rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None
            for sizes in ([40], [20] + [1] * 20):
                assert_close(run_cut(make_engine(cfgd, w, dtype), toks, sizes), ref, dtype, (ls, rs), moves=moves)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype):
    """Five prompts of unlike lengths through ``Engine.generate`` (three slots, prompts cut into portions of 16, a pool
    that holds less than all of them): the tokens are the plain implementation's greedy choices wherever its two best
    logits are further apart than rounding."""
    import cbis_b200 as cb
    cfgd = MIXED if dtype == "float32" else unrouted(MIXED)      # bfloat16: rounding may flip an expert, so none there
    w = make_weights(cfgd, 13)
    prompts = [tokens_of(cfgd, n, 70 + n) for n in (3, 40, 1, 25, 33)]
    new = 12
    opts = dict(num_pages=24, max_num_seqs=3, max_batched_tokens=64, prefill_chunk=16)
    eng = make_engine(cfgd, w, dtype, **opts)
    outs = eng.generate(prompts, cb.SamplingParams(max_new_tokens=new))
    gap = 1e-3 if dtype == "float32" else 0.5
    checked = 0
    for p, o in zip(prompts, outs):
        assert len(o) == new
        seq = list(p)
        for tok in o:
            logits = plain(cfgd, w, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if top2[0] - top2[1] < gap:
                break                                   # a close call: from here on the sequences may part
            assert tok == int(logits.argmax()), (len(p), len(seq))
            seq.append(tok)
            checked += 1
    assert checked >= 5, checked          # some tokens were compared at all
    assert eng.scheduler.idle()
    again = eng.generate(prompts[:2], cb.SamplingParams(max_new_tokens=new))     # slots and pages used again
    assert again == outs[:2]
    warm = make_engine(cfgd, w, dtype, **opts)
    assert warm.warm_up() > 0
    assert warm.generate(prompts[:2], cb.SamplingParams(max_new_tokens=new)) == outs[:2]


def test_sampling_through_the_scheduler_does_not_hang_on_the_batch():
    """Temperature sampling is keyed by request and output index: the same requests give the same tokens whatever
    they are batched with (32-bit)."""
    import cbis_b200 as cb
    w = make_weights(MIXED, 15)
    prompts = [tokens_of(MIXED, n, 20 + n) for n in (9, 17, 4)]
    par = cb.SamplingParams(max_new_tokens=8, temperature=0.8, seed=5)
    one = make_engine(MIXED, w, "float32", max_num_seqs=1).generate(prompts, par)
    assert make_engine(MIXED, w, "float32", max_num_seqs=3).generate(prompts, par) == one


# ---- trace replay through bin/trace_run -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_of_a_model_folder(dtype, tmp_path):
    """A folder (config.json without the sizes that the tensors tell, model.safetensors) through ``bin/trace_run``: a
    request whole; one with its last 20 tokens one by one; one in portions down to two tokens; and four live requests in
    mixed steps through a pool smaller than the requests together, so that pages and request slots are used again."""
    import json
    import os

    from cbis_b200.weights.safetensors_io import write_safetensors
    from replay_helpers import Trace, read_logits, run_trace
    cfgd = MIXED
    w = make_weights(cfgd, 23)
    bare = copy.deepcopy(cfgd)
    for l in bare["layers"]:
        del l["mixer"]["right"]["decay_rank"]
    folder = str(tmp_path / "model")
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(bare, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})
    lens = {"whole": 70, "tail": 50, "cut": 61, "m0": 40, "m1": 33, "m2": 64, "m3": 9, "m4": 21}
    seqs = {r: tokens_of(cfgd, n, 90 + i) for i, (r, n) in enumerate(lens.items())}
    t = Trace()
    t.step([("whole", seqs["whole"], range(70))], end=["whole"])
    t.step([("tail", seqs["tail"][:30], range(30))])
    for i in range(30, 50):
        t.step([("tail", seqs["tail"][i:i + 1], [0])], end=["tail"] if i == 49 else [])
    pos = 0
    for n in [16, 7, 2, 5, 2, 9, 3, 2, 15]:
        t.step([("cut", seqs["cut"][pos:pos + n], range(n))], end=["cut"] if pos + n == 61 else [])
        pos += n
    plan = {"m0": [30, 2, 1, 1, 6], "m1": [2, 20, 1, 10], "m2": [50, 1, 1, 12], "m3": [9], "m4": [3, 1, 17]}
    waiting, live, at, fed = list(plan), [], {}, {}
    while waiting or live:
        while waiting and len(live) < 4:
            r = waiting.pop(0)
            live.append(r)
            at[r] = fed[r] = 0
        entries, ended = [], []
        for r in list(live):
            n = plan[r][at[r]]
            entries.append((r, seqs[r][fed[r]:fed[r] + n], range(n)))
            fed[r] += n
            at[r] += 1
            if at[r] == len(plan[r]):
                ended.append(r)
                live.remove(r)
        t.step(entries, end=ended)
    bound = t.live_tokens_bound()
    assert bound < sum(-(-n // 64) * 64 for n in lens.values())
    out = str(tmp_path / "out")
    run_trace(t, folder, dtype, out, max_tokens=bound, page_size=8, env={"CBIS_POISON_FREED_PAGES": "1"})
    got = read_logits(t, out, cfgd["vocab"])
    for r, toks in seqs.items():
        rows = torch.from_numpy(np.stack([got[(r, p)][0] for p in range(len(toks))])).double()
        ref, _, close = plain_all(cfgd, w, toks)
        assert_close(rows, ref, dtype, r, close, moves=rounding_moves(cfgd, w, toks) if dtype == "bfloat16" else None)
