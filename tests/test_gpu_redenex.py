"""Redenex on the GPU against the plain implementation (tests/redenex_plain.py): each mechanism alone, whole models, prompts in portions,
decoding, batches, pages, slots and states that are used again, the edges of chunks, generation through the serving loop, and the tools."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import redenex_cases as rc
import redenex_plain as rp

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def rt(pkg):
    r = pkg.B200Runtime.initialize(device=0)
    yield r
    r.close()


def load(pkg, rt, tmp_path, cfg, W, dtype, **kw):
    kw.setdefault("max_seq", 512)
    return rt.load_pretrained(rc.save(pkg, tmp_path / "model", cfg, W), dtype=dtype, **kw)


def check(got, want, dtype, factor=1.0):
    """In bf16 single positions may be further off: where the two maps nearly cancel, the norm behind them enlarges their rounding."""
    e, tol = rc.errors(got, want), factor * rc.TOL[dtype]
    assert np.isfinite(got).all() and e.max() < (3 * tol if dtype == "bfloat16" else tol), (int(e.argmax()), float(e.max()))
    assert np.sum(e > tol) <= max(1, 0.05 * e.size), float(np.mean(e > tol))


def both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=150, seed=9, factor=1.0):
    """A prompt in one piece (rows; 150 rows: the tensor-core kernels in bf16) and token by token (decode kernels)."""
    load(pkg, rt, tmp_path, cfg, W, dtype)
    toks = rc.tokens(cfg, n, seed)
    want = rp.forward(cfg, W, toks)
    check(rc.run(rt, toks, [n]), want, dtype, factor)
    check(rc.run(rt, toks, [1]), want, dtype, factor)
    check(rc.run(rt, toks, [n - 20, 5]), want, dtype, factor)


def zero(W, *names):
    for n in names:
        for k in W:
            if k.endswith(n):
                W[k] = np.zeros_like(W[k])
    return W


# ---- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["MIXED", "WIDE"])
def test_prompt_portions_and_decoding(pkg, rt, tmp_path, name, dtype):
    cfg = getattr(rc, name)
    W, toks = rc.weights(cfg, 11), rc.tokens(cfg, 300, 12)
    want = rp.forward(cfg, W, toks)
    load(pkg, rt, tmp_path, cfg, W, dtype)
    for cuts in ([300], [200, 1], [64, 2, 3, 17, 49, 1, 64], [2], [4], [5, 31, 100, 1, 1, 40], [63, 65, 128], [3, 257, 7]):
        check(rc.run(rt, toks, cuts), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_other_sizes(pkg, rt, tmp_path, dtype):
    """Sizes the kernels' tiles do not divide, one stream and eight, loops over everything, over the end and over nothing."""
    for i, (cfg, n) in enumerate([(rc.config([rc.att(1, 1, 6, 3, 1, 7, conv=1), rc.rec(3, 1, 1, conv=1)], width=34, vocab=17, streams=1), 40),
                                  (rc.config([rc.rec(130, 2, 65, conv=6), rc.att(7, 7, 16, 20, 33, None, conv=2)], width=130, vocab=1001, eps=1e-3, streams=8, loop=(0, 2, 2)), 90),
                                  (rc.config([rc.att(5, 5, 30, 9, 21, 27, rot=10), rc.att(3, 1, 18, 45, 64, None), rc.rec(45, 9, 3)], width=45, vocab=30, loop=(2, 3, 4)), 140),
                                  (rc.config([rc.rec(64, 64, None), rc.rec(200, 1, 9, conv=9)], width=64, vocab=64, streams=5, scale=3.0, loop=(1, 1, 5)), 70),
                                  (rc.config([rc.att(24, 1, 96, 64, 40, None, diff=0.0)], width=64, vocab=64, streams=4, loop=(0, 1, 1)), 70),
                                  (rc.config([rc.rec(640, 2, 24), rc.att(2, 1, 144, 160, 100, 24)], width=80, vocab=99, streams=2), 140)]):
        both_ways(pkg, rt, tmp_path / str(i), cfg, rc.weights(cfg, 20 + i), dtype, n)


# ---- mechanisms one at a time: everything else switched off by the weights
ONE_ATT = rc.config([rc.att(4, 2, 24, 16, 40, 72)], width=48, vocab=99)
ONE_REC = rc.config([rc.rec(56, 2, 72)], width=48, vocab=99)


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_norm_and_head(pkg, rt, tmp_path, dtype):
    cfg = {**ONE_ATT, "embedding": {"scale": 12.5}, "norm": {"eps": 0.3}}
    both_ways(pkg, rt, tmp_path, cfg, zero(rc.weights(cfg, 30), "mix.o", "mlp.down"), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 7, 8])
def test_streams(pkg, rt, tmp_path, dtype, streams):
    """Mix matrices far from symmetric, inputs and outputs of both signs."""
    cfg = rc.config([rc.rec(24, 3, 20), rc.att(2, 1, 16, 16, 30, None), rc.rec(24, 3, 20)], width=40, vocab=77, streams=streams)
    W, rng = rc.weights(cfg, 31), np.random.default_rng(32)
    for k in W:
        if ".hc" in k and k.endswith("mix"):
            W[k] = rc.bf16(np.tril(rng.uniform(0.2, 1.0, W[k].shape)) / np.sqrt(streams))
        elif ".hc" in k:
            W[k] = rc.bf16(rng.uniform(-1.5, 1.5, W[k].shape))
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=60)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("limit", [0.25, 1.0, 7.0])
def test_clamped_gate(pkg, rt, tmp_path, dtype, limit):
    cfg = copy.deepcopy(ONE_ATT)
    cfg["layers"][0]["mlp"]["limit"] = limit
    W = zero(rc.weights(cfg, 33), "mix.o")
    for n in ("gate", "up"):
        W["l0.mlp." + n] *= 4.0
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=60)


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrence_alone(pkg, rt, tmp_path, dtype):
    """Channels that forget at once, and channels that remember everything; the gates far into saturation."""
    W = zero(rc.weights(ONE_REC, 34), "mlp.down")
    W["l0.mix.lam"] = rc.bf16(np.tile([-9.0, -6.0, -3.0, 3.0, -12.0, 0.0, 1.0, -7.5], 7))
    W["l0.mix.ra.b"] = rc.bf16(np.random.default_rng(1).uniform(-6, 6, W["l0.mix.ra.b"].shape))
    W["l0.mix.ri.b"] = rc.bf16(np.random.default_rng(2).uniform(-6, 6, W["l0.mix.ri.b"].shape))
    both_ways(pkg, rt, tmp_path, ONE_REC, W, dtype, n=400)


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrence_blocks_do_not_mix(pkg, rt, tmp_path, dtype):
    """Gates of one block large: a block read from its neighbour, or rows and columns exchanged, would show."""
    cfg = rc.config([rc.rec(72, 3, None, conv=2)], width=40, vocab=55, streams=1)
    W = rc.weights(cfg, 35)
    for n in ("ra", "ri"):
        W["l0.mix." + n][1] *= 8.0
        W["l0.mix." + n][2] = np.triu(W["l0.mix." + n][2]) * 2.0
    both_ways(pkg, rt, tmp_path, cfg, W, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_short_convolutions(pkg, rt, tmp_path, dtype, taps):
    """Weights on the oldest tap alone as well: a shift by one, or a ring that is one short, is another token's value."""
    cfg = rc.config([rc.rec(24, 2, None, conv=taps), rc.att(2, 1, 16, 16, None, None, conv=taps)], width=40, vocab=77)
    W = rc.weights(cfg, 36)
    for k in W:
        if k.endswith(".conv"):
            W[k] = np.concatenate([np.ones_like(W[k][:, :1]), np.zeros_like(W[k][:, 1:])], axis=1)
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=70)
    toks = rc.tokens(cfg, 40, 37)
    want = rp.forward(cfg, W, toks)
    for cuts in ([2], [3], [5, 2, 1, 4], [1, 4, 1, 6], [30, 4, 2]):
        check(rc.run(rt, toks, cuts), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot, base", [(2, 10000.0), (10, 40.0), (24, 1000000.0)])
def test_rotation_of_part_of_a_head(pkg, rt, tmp_path, dtype, rot, base):
    cfg = rc.config([rc.att(4, 2, 24, 16, None, None, rot=rot, base=base, scale=1.0)], width=48, vocab=99)
    W = zero(rc.weights(cfg, 38), "q", "k")                    # queries and keys are their biases: the score depends on the distance alone
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=300)


@pytest.mark.parametrize("dtype", DTYPES)
def test_head_norms_and_scale(pkg, rt, tmp_path, dtype):
    """Heads (and maps) of very different sizes: a norm over several of them would hide the small ones."""
    cfg = copy.deepcopy(ONE_ATT)
    cfg["layers"][0]["mixer"].update(scale=0.9, mask=None)
    W = zero(rc.weights(cfg, 39), "mlp.down")
    W["l0.mix.q"][:24] *= 16.0
    W["l0.mix.k"][24:48] *= 1 / 16.0
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, factor=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("diff, size", [(0.0, 1.0), (0.8, 3.0), (0.2, -3.0)])
def test_difference_of_maps(pkg, rt, tmp_path, dtype, diff, size):
    """The second map's weight near 0, large, and negative."""
    cfg = copy.deepcopy(ONE_ATT)
    cfg["layers"][0]["mixer"]["diff"] = diff
    W = zero(rc.weights(cfg, 40, sharp=2.0), "mlp.down")
    v = np.ones(24) / 24
    for n, f in (("lq1", size * 0.5), ("lk1", 1.0), ("lq2", -size * 0.2), ("lk2", 1.0)):
        W["l0.mix." + n] = rc.bf16(f * v * (24 if n[1] == "q" else 1))
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, factor=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [1, 2, 63, 64, 65, 127, 128, 129, 200])
def test_chunk_is_exact(pkg, rt, tmp_path, dtype, size):
    """Uniform weights over the visible keys of map 1 and single keys in map 2: the output counts what it sees."""
    cfg = rc.config([rc.att(6, 2, 32, 32, size, None, conv=1)], width=64, streams=1)
    W = rc.weights(cfg, 41)
    for n in ("q", "q.b"):
        w = W["l0.mix." + n].reshape(6, 2, 32, -1)
        w[:, 0] = 0.0
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=280, factor=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [20, 64, 100, 130])
def test_one_key_stands_out_at_the_edge(pkg, rt, tmp_path, dtype, size):
    """A token whose key scores far above all others (in the first map) is placed at the ends of chunks, pages and tiles: later positions of
    its chunk see it, the first positions of the next do not, in the plain model and on the GPU."""
    cfg = rc.config([rc.att(4, 2, 32, 32, size, None, conv=2, rot=8, scale=0.6)], width=64, streams=1)
    W = rc.weights(cfg, 42)
    rng = np.random.default_rng(43)
    mark, ask = np.linalg.qr(rng.standard_normal((64, 1)))[0][:, 0], np.where(np.arange(32) < 8, 0.0, rng.choice([-1.0, 1.0], 32))
    W["embed"] = rc.bf16(0.5 * (W["embed"] - np.outer(W["embed"] @ mark, mark)))
    W["embed"][5] = rc.bf16(8.0 * mark)
    for c, heads in (("q", 4), ("k", 2)):
        w, b = W[f"l0.mix.{c}"].reshape(heads, 2, 32, 64), W[f"l0.mix.{c}.b"].reshape(heads, 2, 32)
        b[:] = 0.0
        if c == "q":
            b[:, 0] = 4.0 * ask                                # every query asks ...
            w[:, 0] *= 0.3
        else:
            w[:, 0] = 0.3 * w[:, 0] + ask[:, None] * mark      # ... for what the marked token's key holds
        W[f"l0.mix.{c}.conv"][:] = [0.0, 1.0]
        W[f"l0.mix.{c}.norm"][:] = 1.0
    W = {k: rc.bf16(v).reshape(np.shape(v)) for k, v in W.items()}
    for spot in (0, 1, size - 3, size, 63, 64):
        toks = [t if t != 5 else 6 for t in rc.tokens(cfg, 240, 44 + spot)]
        without = list(toks)
        toks[spot] = 5
        want = rp.forward(cfg, W, toks)
        seen = rc.errors(want, rp.forward(cfg, W, without))
        end = (spot // size + 1) * size
        if spot + 2 < end:
            assert seen[min(end, 240) - 1] > 0.3 and (end >= 240 or seen[end:].max() == 0.0)       # it shows, and it is gone
        load(pkg, rt, tmp_path, cfg, W, dtype, kv_page_rows=64)
        for cuts in ([240], [end - 1, 1], [end, 7], [50, 3, 1]):
            check(rc.run(rt, toks, cuts), want, dtype, 1.5)
        rt.kv_release(0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds(pkg, rt, tmp_path, dtype):
    """No chunks: single keys dominate, hundreds of positions back."""
    cfg = rc.config([rc.att(6, 2, 40, 32, None, 40), rc.att(4, 1, 64, 64, 512, 40)], width=72)
    W, toks = rc.weights(cfg, 45, sharp=3.0), rc.tokens(cfg, 700, 46)
    want = rp.forward(cfg, W, toks)
    load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=768)
    for cuts in ([700], [600, 1], [130]):
        check(rc.run(rt, toks, cuts), want, dtype, 2.5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_in_the_state(pkg, rt, tmp_path, dtype):
    """The first token alone drives a slow state; hundreds of tokens later it is still there, through portions and single steps."""
    cfg = rc.config([rc.rec(64, 2, None)], width=48, vocab=99, streams=2)
    W = rc.weights(cfg, 47)
    W["l0.mix.lam"][:] = rc.bf16(-10.0)
    W["embed"] = rc.bf16(W["embed"] * 0.05)
    W["embed"][7] = rc.bf16(W["embed"][7] * 200)
    W["l0.mix.x.b"][:] = 0.0
    W["l0.mix.conv.b"][:] = 0.0
    cfg["norm"]["eps"] = 1.0
    toks = [7] + [t if t != 7 else 8 for t in rc.tokens(cfg, 599, 48)]
    want = rp.forward(cfg, W, toks)
    assert rc.errors(want, rp.forward(cfg, W, [8] + toks[1:]))[500:].min() > 0.02
    load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=640)
    for cuts in ([600], [400, 1], [100, 2, 64, 1]):
        check(rc.run(rt, toks, cuts), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(pkg, rt, tmp_path, dtype):
    W = rc.weights(rc.MIXED, 49)
    load(pkg, rt, tmp_path, rc.MIXED, W, dtype)
    rc.run(rt, rc.tokens(rc.MIXED, 60, 1), [60])               # (a used slot)
    for n in (1, 2, 3, 4, 5, 15, 16, 17):
        toks = rc.tokens(rc.MIXED, n, n)
        check(rc.run(rt, toks, [n]), rp.forward(rc.MIXED, W, toks), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_loops_keep_passes_apart(pkg, rt, tmp_path, dtype):
    for i, loop in enumerate([None, (0, 3, 2), (1, 2, 4), (1, 3, 1), (2, 3, 3)]):
        cfg = rc.config([rc.rec(24, 3, 20), rc.att(2, 1, 16, 16, 30, 24), rc.rec(24, 2, None)], width=40, vocab=77, loop=loop)
        both_ways(pkg, rt, tmp_path / str(i), cfg, rc.weights(cfg, 50 + i), dtype, n=80)


# ---- cache and state: slots, pages, batches
@pytest.mark.parametrize("pages", [0, 64])
def test_slots_and_pages_used_again(pkg, rt, tmp_path, pages):
    cfg, dtype = rc.MIXED, "float32"
    W = rc.weights(cfg, 55)
    kw = dict(max_seq=256, max_batch=3)
    if pages:
        kw.update(kv_page_rows=pages, kv_pool_pages=7)
    load(pkg, rt, tmp_path, cfg, W, dtype, **kw)
    for turn, n in enumerate((200, 70, 130, 5, 250)):
        slot, toks = turn % 3, rc.tokens(cfg, n, 56 + turn)
        check(rc.run(rt, toks, [n // 2 + 1, 1, 9], slot=slot), rp.forward(cfg, W, toks), dtype)
        rt.kv_release(slot)
    if pages:
        assert rt.kv_pool() == (7, 7, 64)


@pytest.mark.parametrize("dtype", DTYPES)
def test_contiguous_and_paged_agree_bit_for_bit(pkg, rt, tmp_path, dtype):
    cfg = rc.WIDE
    W, toks, got = rc.weights(cfg, 60), rc.tokens(cfg, 200, 61), []
    for pages in (0, 64, 128):
        load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=256, max_batch=2, kv_page_rows=pages)
        if pages:
            rt.seq_select(0); rt.set_data(toks[:70]); rt.execute({"s": 70, "p": 0})       # pages of sequence 1 do not start at 0
        got.append(rc.run(rt, toks, [150, 1], slot=1))
    assert np.array_equal(got[0], got[1]) and np.array_equal(got[0], got[2])


def test_interleaved_requests(pkg, rt, tmp_path):
    """Portions of three requests in turn, one of them restarted in a slot that was used: each as if alone."""
    cfg, dtype = rc.MIXED, "float32"
    W = rc.weights(cfg, 62)
    load(pkg, rt, tmp_path, cfg, W, dtype, **pkg.replay.TraceReplay.capacity(600, 4))
    r = pkg.replay.TraceReplay(rt, 4)
    reqs = {"a": rc.tokens(cfg, 180, 1), "b": rc.tokens(cfg, 9, 2), "c": rc.tokens(cfg, 111, 3), "a2": rc.tokens(cfg, 180, 1)}
    at, got, rng = {k: 0 for k in reqs}, {k: [] for k in reqs}, np.random.default_rng(5)
    live = ["a", "b", "c"]
    while live:
        k = live[int(rng.integers(len(live)))]
        n = int(min(rng.integers(1, 50), len(reqs[k]) - at[k]))
        end = [k] if at[k] + n == len(reqs[k]) else []
        got[k] += r.step([{"id": k, "tokens": reqs[k][at[k]:at[k] + n], "want": list(range(n))}], end)
        at[k] += n
        if end:
            live.remove(k)
            if k == "b":
                live.append("a2")
    for k, toks in reqs.items():
        check(np.stack(got[k]), rp.forward(cfg, W, toks), dtype)
    assert rt.kv_pool()[0] == rt.kv_pool()[1]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pages", [0, 64])
def test_batch_of_unequal_requests(pkg, rt, tmp_path, dtype, pages):
    """Batched steps over sequences of very different lengths equal each one alone (the batch takes other kernels: up to rounding)."""
    for j, cfg in enumerate((rc.MIXED, rc.WIDE)):
        W = rc.weights(cfg, 63)
        load(pkg, rt, tmp_path / str(j), cfg, W, dtype, max_seq=256, max_batch=5, kv_page_rows=pages)
        prompts = [rc.tokens(cfg, n, 60 + n) for n in (3, 64, 150, 1, 33)]
        slots, cur = [4, 0, 2, 1, 3], []
        for s, p in zip(slots, prompts):
            rt.seq_select(s); rt.set_data(p); rt.execute({"s": len(p), "p": 0})
            cur.append(rt.get_token())
        for _ in range(7):                                     # (more steps than a convolution has taps)
            rt.batch_begin_slots(slots, cur, [len(p) for p in prompts])
            rt.batch_decode(1)
            nxt = rt.batch_get_decoded(1)[0]
            for i, p in enumerate(prompts):
                p.append(int(cur[i]))
                check(rt.batch_get_logits(i)[None], rp.forward(cfg, W, p, rows=[len(p) - 1]), dtype, 1.5)
            cur = [int(t) for t in nxt]
        p, s = prompts[2], slots[2]                            # and on alone, from the state the batch left
        more = rc.tokens(cfg, 20, 64)
        check(rc.run(rt, more, [1, 6], slot=s, start=len(p)), rp.forward(cfg, W, p + more)[len(p):], dtype, 1.5)


def test_state_is_guarded_saved_and_copied(pkg, rt, tmp_path):
    cfg, dtype = rc.MIXED, "float32"
    W, toks = rc.weights(cfg, 65), rc.tokens(cfg, 90, 66)
    want = rp.forward(cfg, W, toks)
    runs = rp.layer_order(len(cfg["layers"]), cfg["loop"])
    load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=128, max_batch=3)
    check(rc.run(rt, toks[:50], [50]), want[:50], dtype)
    for p in (49, 51, 3):                                      # the state stands at 50
        rt.set_data(toks[:2])
        with pytest.raises(pkg.LumError):
            rt.execute({"s": 2, "p": p})
    with pytest.raises(pkg.LumError):
        rt.kv_copy(0, 1, 49)
    with pytest.raises(pkg.LumError):
        rt.batch_begin_slots([0, 1], [1, 2], [49, 0])
    rt.profile(3)                                              # trial steps leave the sequence where it was
    rt.kv_copy(0, 1, 50)
    state, pos = rt.state_save()
    assert pos == 50 and state.size > 0
    saved = [(i, k, rt.kv_save(i, k, 50)) for i in range(len(runs)) for k in ("k", "v")]
    check(rc.run(rt, toks[50:], [7, 1], slot=0, start=50), want[50:], dtype)
    check(rc.run(rt, toks[50:], [30, 4], slot=1, start=50), want[50:], dtype)
    rt.kv_reset()
    rt.seq_select(2)
    for i, k, data in saved:
        rt.kv_load(i, k, 50, data)
    rt.state_load(state, pos)
    check(rc.run(rt, toks[50:], [3, 20], slot=2, start=50), want[50:], dtype)


# ---- generation
def greedy(cfg, W, prompt, n):
    """Plain greedy generation; also the smallest margin between the two best logits on the way."""
    toks, margin = list(prompt), np.inf
    for _ in range(n):
        lg = rp.forward(cfg, W, toks, rows=[len(toks) - 1])[0]
        top = np.sort(lg)[-2:]
        margin = min(margin, (top[1] - top[0]) / lg.std())
        toks.append(int(lg.argmax()))
    return toks[len(prompt):], margin


def test_greedy_generation_and_serving_loop(pkg, rt, tmp_path):
    cfg = rc.MIXED
    W = rc.weights(cfg, 70)
    load(pkg, rt, tmp_path, cfg, W, "float32", max_seq=192, max_batch=3, kv_page_rows=64)
    prompts = [rc.tokens(cfg, n, 71 + n) for n in (20, 3, 70, 1, 40)]
    want = [greedy(cfg, W, p, 24) for p in prompts]
    assert min(m for _, m in want) > 1e-4                      # (no near ties: rounding cannot change the choice)
    assert [int(t) for t in rt.generate(prompts[0], 24)] == want[0][0]
    rt.kv_reset()
    b = pkg.serving.ContinuousBatcher(rt, steps_per_round=5)
    ids = [b.submit(p, 24) for p in prompts]
    out = b.run()
    assert [out[i] for i in ids] == [w for w, _ in want]
    rt.kv_reset()
    b = pkg.serving.ContinuousBatcher(rt, steps_per_round=4)   # a prefix computed once: its rows and its state
    b.park_prefix(prompts[2][:50])
    ids = [b.submit(p, 24) for p in (prompts[2], prompts[1], prompts[2])]
    out = b.run()
    assert [out[i] for i in ids] == [want[2][0], want[1][0], want[2][0]]
    assert [b.finished[i].reused_rows for i in ids] == [50, 0, 50]


def test_sampling(pkg, rt, tmp_path):
    cfg = rc.WIDE
    load(pkg, rt, tmp_path, cfg, rc.weights(cfg, 72), "bfloat16", max_seq=256, max_batch=4, kv_page_rows=64)
    rt.set_sampling(0.9, 40, 0.95, 7)
    p = rc.tokens(cfg, 30, 73)
    a = rt.generate(p, 12)
    assert a == rt.generate(p, 12) and all(0 <= t < cfg["vocab"] for t in a)
    rt.set_sampling(0.0)


def test_long_decoding(pkg, rt, tmp_path):
    cfg = rc.MIXED
    W, toks = rc.weights(cfg, 74), rc.tokens(cfg, 500, 75)
    load(pkg, rt, tmp_path, cfg, W, "float32", max_seq=512)
    check(rc.run(rt, toks, [10, 1]), rp.forward(cfg, W, toks), "float32")


# ---- weights through the C ABI
@pytest.mark.parametrize("dtype", DTYPES)
def test_weights_round_trip(pkg, rt, tmp_path, dtype):
    cfg = rc.MIXED
    W = rc.weights(cfg, 80)
    load(pkg, rt, tmp_path, cfg, W, dtype)
    for slot, layer, name in [("q", 1, "l1.mix.q"), ("k", 3, "l3.mix.k"), ("v_conv", 4, "l4.mix.v.conv"), ("o", 0, "l0.mix.o"), ("gate", 1, "l1.mlp.gate"), ("up", 5, "l5.mlp.up"),
                              ("down", 4, "l4.mlp.down"), ("rec_ra", 0, "l0.mix.ra"), ("rec_ri", 2, "l2.mix.ri"), ("rec_x_bias", 0, "l0.mix.x.b"), ("hc2_mix", 1, "l1.hc2.mix"),
                              ("k_bias", 5, "l5.mix.k.b"), ("rec_lam", 2, "l2.mix.lam"), ("lk2", 4, "l4.mix.lk2"), ("mlp_norm", 0, "l0.norm2")]:
        assert np.array_equal(rt.get_weight_f32(slot, layer, 0, W[name].size), W[name].ravel()), name
    rt.save_safetensors(str(tmp_path / "shard.safetensors"))
    toks = rc.tokens(cfg, 40, 81)
    first = rc.run(rt, toks, [40])
    spec = pkg.models.from_config(cfg, dtype=dtype, max_seq=64)
    rt.load_model(spec.desc, spec.layers)
    loaded, ignored = rt.load_safetensors(str(tmp_path / "shard.safetensors"))
    assert (loaded, ignored) == (len(spec.tensor_names()), 0)
    assert np.array_equal(rc.run(rt, toks, [40]), first)


def test_descriptors_the_runtime_does_not_have_are_refused(pkg, rt):
    for change in (dict(streams=9), dict(loop_start=3, loop_stop=9, loop_times=2), dict(norm_kind=1), dict(tied_head=1)):
        spec = pkg.models.from_config(rc.MIXED)
        for k, v in change.items():
            setattr(spec.desc, k, v)
        with pytest.raises(pkg.LumError):
            rt.load_model(spec.desc, spec.layers)
    for change in (dict(maps=3), dict(rot_dims=7), dict(conv_taps=-1), dict(ffn_kind=0), dict(mixer=2)):
        spec = pkg.models.from_config(rc.MIXED)
        for k, v in change.items():
            setattr(spec.layers[1], k, v)
        with pytest.raises(pkg.LumError):
            rt.load_model(spec.desc, spec.layers)


def test_one_residual_vector_without_streams(pkg, rt):
    """streams 0 is the ordinary residual sum: the same as one stream whose three numbers are 1."""
    cfg = rc.config([rc.rec(24, 3, 20), rc.att(2, 1, 16, 16, 30, 24)], width=40, vocab=77, streams=1)
    W, toks, got = rc.weights(cfg, 82), rc.tokens(cfg, 50, 83), []
    for streams in (1, 0):
        spec = pkg.models.from_config(cfg, dtype="float32", max_seq=64)
        spec.desc.streams = streams
        rt.load_model(spec.desc, spec.layers)
        for name in spec.tensor_names():
            rt.set_weight(*SLOT_OF(pkg, name), np.ones_like(W[name]) if ".hc" in name else W[name], "f32")
        got.append((rc.run(rt, toks, [40, 1]), rc.run(rt, toks, [1])))
    one = {k: np.ones_like(v) if ".hc" in k else v for k, v in W.items()}
    check(got[0][0], rp.forward(cfg, one, toks), "float32")
    for a, b in zip(got[0], got[1]):
        assert np.array_equal(a, b)


def SLOT_OF(pkg, name):
    names = {"embed": "embed", "final.norm": "final_norm", "head": "lm_head", "norm1": "attn_norm", "norm2": "mlp_norm", "mix.o": "o", "mlp.gate": "gate", "mlp.up": "up",
             "mlp.down": "down", "mix.y": "rec_y", "mix.y.b": "rec_y_bias", "mix.x": "rec_x", "mix.x.b": "rec_x_bias", "mix.conv": "rec_conv", "mix.conv.b": "rec_conv_bias",
             "mix.ra": "rec_ra", "mix.ra.b": "rec_ra_bias", "mix.ri": "rec_ri", "mix.ri.b": "rec_ri_bias", "mix.lam": "rec_lam"}
    names.update({f"mix.{c}{s}": f"{c}{t}" for c in "qkv" for s, t in (("", ""), (".b", "_bias"), (".conv", "_conv"), (".norm", "_norm"))})
    names.update({f"mix.{c}": c for c in ("lq1", "lk1", "lq2", "lk2")})
    names.update({f"hc{q}.{n}": f"hc{q}_{n}" for q in (1, 2) for n in ("in", "out", "mix")})
    if name in names:
        return names[name], 0
    layer, rest = name.split(".", 1)
    return names[rest], int(layer[1:])


# ---- the tools
@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run(pkg, tmp_path, dtype):
    cfg = rc.MIXED
    W = rc.weights(cfg, 90)
    folder = rc.save(pkg, tmp_path / "m", cfg, W)
    out = tmp_path / "out"
    out.mkdir()
    toks = rc.tokens(cfg, 90, 91)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:80], "want": [79, 3]}], "end": []}, {"step": 1, "entries": [{"id": "x", "tokens": toks[80:88], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[88:], "want": [0, 1]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "90"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = rp.forward(cfg, W, toks)
    assert not (out / "1.f32").exists()
    check(np.fromfile(out / "0.f32", "<f4").reshape(2, -1), want[[79, 3]], dtype)
    check(np.fromfile(out / "2.f32", "<f4").reshape(2, -1), want[[88, 89]], dtype)


def test_generate_tool(pkg, tmp_path):
    cfg = rc.MIXED
    W = rc.weights(cfg, 70)
    folder = rc.save(pkg, tmp_path / "m", cfg, W)
    prompts = [rc.tokens(cfg, n, 71 + n) for n in (20, 3)]
    cmd = [sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", folder, "--dtype", "float32", "--max-new", "6", "--max-seq", "128"]
    for p in prompts:
        cmd += ["--prompt", ",".join(map(str, p))]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    for line, p in zip(r.stdout.splitlines(), prompts):
        assert json.loads(line) == {"prompt": p, "tokens": greedy(cfg, W, p, 6)[0]}
