"""Madipel on the GPU against the plain implementation (tests/madipel_plain.py): each mechanism alone, whole models, prompts in portions,
decoding, batches, pages and slots that are used again, the far ends of windows, generation through the serving loop, and the tools."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import madipel_cases as mc
import madipel_plain as mp

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
    return rt.load_pretrained(mc.save(pkg, tmp_path / "model", cfg, W), dtype=dtype, **kw)


def check(got, want, dtype, factor=1.0):
    e = mc.errors(got, want)
    assert np.isfinite(got).all() and e.max() < factor * mc.TOL[dtype], (int(e.argmax()), float(e.max()))


def both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=150, seed=9, factor=1.0):
    """A prompt in one piece (rows; 150 rows: the tensor-core kernels in bf16) and token by token (decode kernels)."""
    load(pkg, rt, tmp_path, cfg, W, dtype)
    toks = mc.tokens(cfg, n, seed)
    want = mp.forward(cfg, W, toks)
    check(mc.run(rt, toks, [n]), want, dtype, factor)
    check(mc.run(rt, toks, [1]), want, dtype, factor)


# ---- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["MIXED", "WIDE"])
def test_prompt_portions_and_decoding(pkg, rt, tmp_path, name, dtype):
    cfg = getattr(mc, name)
    W, toks = mc.weights(cfg, 11), mc.tokens(cfg, 300, 12)
    want = mp.forward(cfg, W, toks)
    load(pkg, rt, tmp_path, cfg, W, dtype)
    for cuts in ([300], [200, 1], [64, 2, 3, 17, 49, 1, 64], [2], [5, 31, 100, 1, 1, 40], [63, 65, 128]):
        check(mc.run(rt, toks, cuts), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_other_sizes(pkg, rt, tmp_path, dtype):
    """One layer, sizes the kernels' tiles do not divide: one head, equal head counts, widths of 34 and 45, a single-token window."""
    for i, (cfg, n) in enumerate([(mc.config([mc.layer(1, 1, 5, 3, 1, 7)], width=34, vocab=17), 40),
                                  (mc.config([mc.layer(7, 7, 16, 20, 33, 65), mc.layer(7, 7, 8, 20, 2, 1)], width=130, vocab=1001, eps=1e-3), 90),
                                  (mc.config([mc.layer(5, 5, 31, 9, 21, 27), mc.layer(3, 1, 17, 45, 64, None)], width=45, vocab=30), 140),
                                  (mc.config([mc.layer(24, 1, 96, 64, 40, None, mix=False)], width=64, vocab=64, mult=2.0), 70)]):
        both_ways(pkg, rt, tmp_path / str(i), cfg, mc.weights(cfg, 20 + i), dtype, n)


# ---- mechanisms one at a time: everything else switched off by the weights
ONE = mc.config([mc.layer(4, 2, 24, 16, 40, 72)], width=48, vocab=99, mult=0.8, logit_scale=1.5)


def zero(W, *names):
    for n in names:
        for k in W:
            if k.endswith(n):
                W[k] = np.zeros_like(W[k])
    return W


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_positions_norm_and_head(pkg, rt, tmp_path, dtype):
    W = zero(mc.weights(ONE, 30), "mix.o", "mlp.down")
    W["embed"] *= 0.25          # (the sinusoid is the larger part)
    both_ways(pkg, rt, tmp_path, ONE, W, dtype, n=400)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("p, q", [(0.0, 0.0), (3.0, -4.0), (-6.0, 2.5), (30.0, -30.0)])
def test_activation(pkg, rt, tmp_path, dtype, p, q):
    W = zero(mc.weights(ONE, 31), "mix.o")
    W["l0.mlp.act"] = mc.bf16([p, q])
    W["l0.mlp.up"] *= 2.0
    both_ways(pkg, rt, tmp_path, ONE, W, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_norm_removes_the_mean(pkg, rt, tmp_path, dtype):
    W = mc.weights(ONE, 32)
    W["embed"] = mc.bf16(W["embed"] + 20.0)
    both_ways(pkg, rt, tmp_path, ONE, W, dtype, factor=4.0)      # (the residual stream's own rounding is larger at this offset)


@pytest.mark.parametrize("dtype", DTYPES)
def test_query_and_key_norms_span_all_heads(pkg, rt, tmp_path, dtype):
    """One head's projection is much larger than the others': a norm per head would hide that."""
    W = mc.weights(ONE, 33, sharp=2.0)
    W["l0.mix.q"][:24] *= 16.0
    W["l0.mix.k"][24:] *= 16.0
    zero(W, "mlp.down")
    both_ways(pkg, rt, tmp_path, ONE, W, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_distance_bias_alone(pkg, rt, tmp_path, dtype):
    W = zero(mc.weights(ONE, 34), "q.norm", "mlp.down")          # scores are the bias alone
    W["l0.mix.r1"] = mc.bf16([0.02, 0.5, 2.5, 1.0])
    W["l0.mix.r2"] = mc.bf16([0.5, 8.0, 0.05, 1.0])
    both_ways(pkg, rt, tmp_path, ONE, W, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_temperature_and_scale_alone(pkg, rt, tmp_path, dtype):
    cfg = copy.deepcopy(ONE)
    cfg["layers"][0]["mixer"]["scale"] = 0.7
    W = zero(mc.weights(cfg, 35), "mix.r1", "mlp.down")
    W["l0.mix.temp"] = mc.bf16([0.0, 0.25, 1.0, 3.0])
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, factor=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_value_mixing(pkg, rt, tmp_path, dtype):
    """Layers without mixing before, between and behind; shares of 0, 1, beyond 1 and below 0; the first mixing layer's own number unused."""
    for lams in ([9.0, 0.0, 1.0], [0.5, 1.5, -0.25]):
        cfg = mc.config([mc.layer(4, 2, 24, 16, 40, None, mix=False), mc.layer(4, 2, 24, 16, 40, 30), mc.layer(2, 1, 16, 32, 40, 30),
                         mc.layer(4, 4, 24, 24, 9, None, mix=False), mc.layer(8, 8, 16, 4, 40, None)], width=48)
        W = mc.weights(cfg, 36)
        for i, v in zip((1, 2, 4), lams):
            W[f"l{i}.mix.vmix"] = mc.bf16(v).reshape(())
        both_ways(pkg, rt, tmp_path / str(lams[0]), cfg, W, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 127, 128, 129, 200])
def test_window_is_exact(pkg, rt, tmp_path, dtype, window):
    """Uniform weights over the window: the output counts the keys it sees."""
    cfg = mc.config([mc.layer(6, 2, 32, 32, window, None)], width=64, mult=3.0)
    W = zero(mc.weights(cfg, 37), "q.norm", "mix.r1")
    both_ways(pkg, rt, tmp_path, cfg, W, dtype, n=280)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [20, 64, 100, 130])
def test_one_key_stands_out_at_the_edge(pkg, rt, tmp_path, dtype, window):
    """A token whose key scores far above all others is placed so that later positions see it just inside and just outside their window, and
    at the borders of pages and tiles; the plain model's logits jump where it leaves the window, and the GPU's jump there too."""
    cfg = mc.config([mc.layer(4, 2, 32, 32, window, None)], width=64, mult=1.0)
    W = mc.weights(cfg, 38)
    W["l0.mix.r1"] *= 0.05
    rng = np.random.default_rng(39)
    mark, ask = np.linalg.qr(rng.standard_normal((64, 2)))[0].T * 8.0
    W["embed"] = mc.bf16(0.3 * W["embed"])
    W["embed"][5] = mc.bf16(6.0 * mark)                      # a token of its own direction, which the keys pick up ...
    W["l0.mix.k"] = mc.bf16(0.3 * W["l0.mix.k"] + np.outer(np.ones(64), mark) / 64)
    W["l0.norm1.b"] = mc.bf16(0.5 * ask)                     # ... while every query asks for what such a key holds
    W["l0.mix.q"] = mc.bf16(0.3 * W["l0.mix.q"] + np.outer(np.ones(128), ask) / 16)
    W["l0.mix.q.norm"] = np.full(128, 3.0, np.float32)
    W["l0.mix.k.norm"] = np.ones(64, np.float32)
    for spot in (0, 1, 63, 64, 70):
        toks = [t if t != 5 else 6 for t in mc.tokens(cfg, 240, 40 + spot)]
        without = list(toks)
        toks[spot] = 5
        want, other = mp.forward(cfg, W, toks), mp.forward(cfg, W, without)
        seen = mc.errors(want, other)
        assert seen[spot + window - 1] > 0.3 and (spot + window >= 240 or seen[spot + window] == 0.0)       # it shows, and it is gone
        load(pkg, rt, tmp_path, cfg, W, dtype, kv_page_rows=64)
        for cuts in ([240], [spot + window - 1 or 1, 1], [spot + window, 7], [50, 3, 1]):
            check(mc.run(rt, toks, cuts), want, dtype, 1.5)
        rt.kv_release(0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds(pkg, rt, tmp_path, dtype):
    """No window: single keys dominate, hundreds of positions back."""
    cfg = mc.config([mc.layer(6, 2, 40, 32, None, 40), mc.layer(4, 1, 64, 64, None, 40)], width=72)
    W = mc.weights(cfg, 41, sharp=3.0)
    for k in W:
        if k.endswith("mix.r1"):
            W[k] = mc.bf16(W[k] * 0.02)
    toks = mc.tokens(cfg, 700, 42)
    want = mp.forward(cfg, W, toks)
    load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=768)
    check(mc.run(rt, toks, [700]), want, dtype, 2.0)
    check(mc.run(rt, toks, [600, 1]), want, dtype, 2.0)
    check(mc.run(rt, toks, [130]), want, dtype, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(pkg, rt, tmp_path, dtype):
    W = mc.weights(mc.MIXED, 43)
    load(pkg, rt, tmp_path, mc.MIXED, W, dtype)
    for n in (1, 2, 3, 4, 5, 15, 16, 17):
        toks = mc.tokens(mc.MIXED, n, n)
        check(mc.run(rt, toks, [n]), mp.forward(mc.MIXED, W, toks), dtype)


# ---- cache: slots, pages, batches
@pytest.mark.parametrize("pages", [0, 64])
def test_slots_and_pages_used_again(pkg, rt, tmp_path, pages):
    cfg, dtype = mc.MIXED, "float32"
    W = mc.weights(cfg, 44)
    kw = dict(max_seq=256, max_batch=3)
    if pages:
        kw.update(kv_page_rows=pages, kv_pool_pages=7)
    load(pkg, rt, tmp_path, cfg, W, dtype, **kw)
    for turn, n in enumerate((200, 70, 130, 5, 250)):
        slot, toks = turn % 3, mc.tokens(cfg, n, 50 + turn)
        check(mc.run(rt, toks, [n // 2 + 1, 1, 9], slot=slot), mp.forward(cfg, W, toks), dtype)
        rt.kv_release(slot)
    if pages:
        assert rt.kv_pool() == (7, 7, 64)


@pytest.mark.parametrize("dtype", DTYPES)
def test_contiguous_and_paged_agree_bit_for_bit(pkg, rt, tmp_path, dtype):
    cfg = mc.WIDE
    W, toks, got = mc.weights(cfg, 45), mc.tokens(cfg, 200, 46), []
    for pages in (0, 64, 128):
        load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=256, max_batch=2, kv_page_rows=pages)
        if pages:
            rt.seq_select(0); rt.set_data(toks[:70]); rt.execute({"s": 70, "p": 0})       # pages of sequence 1 do not start at 0
        got.append(mc.run(rt, toks, [150, 1], slot=1))
    assert np.array_equal(got[0], got[1]) and np.array_equal(got[0], got[2])


def test_interleaved_requests(pkg, rt, tmp_path):
    """Portions of three requests in turn, one of them restarted in a slot that was used: each as if alone."""
    cfg, dtype = mc.MIXED, "float32"
    W = mc.weights(cfg, 47)
    load(pkg, rt, tmp_path, cfg, W, dtype, **pkg.replay.TraceReplay.capacity(600, 4))
    r = pkg.replay.TraceReplay(rt, 4)
    reqs = {"a": mc.tokens(cfg, 180, 1), "b": mc.tokens(cfg, 9, 2), "c": mc.tokens(cfg, 111, 3), "a2": mc.tokens(cfg, 180, 1)}
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
        check(np.stack(got[k]), mp.forward(cfg, W, toks), dtype)
    assert rt.kv_pool()[0] == rt.kv_pool()[1]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pages", [0, 64])
def test_batch_of_unequal_requests(pkg, rt, tmp_path, dtype, pages):
    """Batched steps over sequences of very different lengths equal each one alone (the batch takes other kernels: up to rounding)."""
    cfg = mc.MIXED
    W = mc.weights(cfg, 48)
    load(pkg, rt, tmp_path, cfg, W, dtype, max_seq=256, max_batch=5, kv_page_rows=pages)
    prompts = [mc.tokens(cfg, n, 60 + n) for n in (3, 64, 150, 1, 33)]
    slots, cur = [4, 0, 2, 1, 3], []
    for s, p in zip(slots, prompts):
        rt.seq_select(s); rt.set_data(p); rt.execute({"s": len(p), "p": 0})
        cur.append(rt.get_token())
    for _ in range(2):
        rt.batch_begin_slots(slots, cur, [len(p) for p in prompts])
        rt.batch_decode(1)
        nxt = rt.batch_get_decoded(1)[0]
        for i, p in enumerate(prompts):
            p.append(int(cur[i]))
            check(rt.batch_get_logits(i)[None], mp.forward(cfg, W, p, rows=[len(p) - 1]), dtype, 1.5)
        cur = [int(t) for t in nxt]


# ---- generation
def greedy(cfg, W, prompt, n):
    """Plain greedy generation; also the smallest margin between the two best logits on the way."""
    toks, margin = list(prompt), np.inf
    for _ in range(n):
        lg = mp.forward(cfg, W, toks, rows=[len(toks) - 1])[0]
        top = np.sort(lg)[-2:]
        margin = min(margin, (top[1] - top[0]) / lg.std())
        toks.append(int(lg.argmax()))
    return toks[len(prompt):], margin


def test_greedy_generation_and_serving_loop(pkg, rt, tmp_path):
    cfg = mc.MIXED
    W = mc.weights(cfg, 70)
    load(pkg, rt, tmp_path, cfg, W, "float32", max_seq=192, max_batch=3, kv_page_rows=64)
    prompts = [mc.tokens(cfg, n, 71 + n) for n in (20, 3, 70, 1, 40)]
    want = [greedy(cfg, W, p, 24) for p in prompts]
    assert min(m for _, m in want) > 1e-4                      # (no near ties: rounding cannot change the choice)
    assert [int(t) for t in rt.generate(prompts[0], 24)] == want[0][0]
    rt.kv_reset()
    b = pkg.serving.ContinuousBatcher(rt, steps_per_round=5)
    ids = [b.submit(p, 24) for p in prompts]
    out = b.run()
    assert [out[i] for i in ids] == [w for w, _ in want]


def test_shared_prefix_and_sampling(pkg, rt, tmp_path):
    cfg = mc.WIDE
    W = mc.weights(cfg, 72)
    prefix = mc.tokens(cfg, 75, 73)
    outs = []
    for park in (False, True):
        load(pkg, rt, tmp_path, cfg, W, "bfloat16", max_seq=256, max_batch=4, kv_page_rows=64)
        rt.set_sampling(0.0)
        b = pkg.serving.ContinuousBatcher(rt)
        if park:
            b.park_prefix(prefix)
        ids = [b.submit(prefix + mc.tokens(cfg, n, n), 8) for n in (4, 20)]
        out = b.run()
        outs.append([out[i] for i in ids])
    same = sum(x == y for a, c in zip(*outs) for x, y in zip(a, c))
    assert same >= 8                                           # (bf16: another cut of the prompt may flip a near tie)
    rt.set_sampling(0.9, 40, 0.95, 7)
    a = rt.generate(prefix[:30], 12)
    assert a == rt.generate(prefix[:30], 12) and all(0 <= t < cfg["vocab"] for t in a)
    rt.set_sampling(0.0)


def test_long_decoding(pkg, rt, tmp_path):
    cfg = mc.MIXED
    W, toks = mc.weights(cfg, 74), mc.tokens(cfg, 500, 75)
    want = mp.forward(cfg, W, toks)
    load(pkg, rt, tmp_path, cfg, W, "float32", max_seq=512)
    check(mc.run(rt, toks, [10, 1]), want, "float32")


# ---- weights and cache through the C ABI
@pytest.mark.parametrize("dtype", DTYPES)
def test_weights_round_trip(pkg, rt, tmp_path, dtype):
    cfg = mc.MIXED
    W = mc.weights(cfg, 80)
    load(pkg, rt, tmp_path, cfg, W, dtype)
    for slot, layer, name in [("q", 0, "l0.mix.q"), ("k", 3, "l3.mix.k"), ("v", 1, "l1.mix.v"), ("o", 2, "l2.mix.o"), ("up", 2, "l2.mlp.up"),
                              ("down", 3, "l3.mlp.down"), ("lm_head", 0, "head"), ("dist_r2", 2, "l2.mix.r2"), ("act", 0, "l0.mlp.act"), ("v_mix", 1, "l1.mix.vmix")]:
        assert np.array_equal(rt.get_weight_f32(slot, layer, 0, W[name].size), W[name].ravel()), name
    rt.save_safetensors(str(tmp_path / "shard.safetensors"))
    toks = mc.tokens(cfg, 40, 81)
    first = mc.run(rt, toks, [40])
    spec = pkg.models.from_config(cfg, dtype=dtype, max_seq=64)
    rt.load_model(spec.desc, spec.layers)
    loaded, ignored = rt.load_safetensors(str(tmp_path / "shard.safetensors"))
    assert (loaded, ignored) == (len(spec.tensor_names()), 0)
    assert np.array_equal(mc.run(rt, toks, [40]), first)


def test_cache_rows_can_be_parked(pkg, rt, tmp_path):
    cfg = mc.MIXED
    W, toks = mc.weights(cfg, 82), mc.tokens(cfg, 60, 83)
    load(pkg, rt, tmp_path, cfg, W, "bfloat16", max_seq=128, max_batch=2)
    whole = mc.run(rt, toks, [40, 20])[40:]
    saved = [(l, k, rt.kv_save(l, k, 40)) for l in range(4) for k in ("k", "v")]
    assert rt.kv_read(3, "k", 40).shape == (40, 2 * 48)
    rt.kv_reset()
    rt.seq_select(1)
    for l, k, data in saved:
        rt.kv_load(l, k, 40, data)
    assert np.array_equal(mc.run(rt, toks[40:], [20], slot=1, start=40), whole)


def test_bad_calls_are_refused(pkg, rt, tmp_path):
    cfg = mc.MIXED
    load(pkg, rt, tmp_path, cfg, mc.weights(cfg, 84), "bfloat16", max_seq=64)
    with pytest.raises(pkg.LumError):
        rt.want_logits([3, 1])
    rt.want_logits([5])
    rt.set_data([1, 2])
    with pytest.raises(pkg.LumError):
        rt.execute({"s": 2, "p": 0})
    spec = pkg.models.from_config(cfg)
    with pytest.raises(pkg.LumError):
        rt.load_model(spec.desc)                               # layers missing
    bad = copy.deepcopy(cfg)
    bad["layers"][3]["mixer"]["vdim"] = 20                     # value widths of mixing layers differ
    spec = pkg.models.from_config(bad)
    with pytest.raises(pkg.LumError):
        rt.load_model(spec.desc, spec.layers)


def test_logits_of_chosen_rows_of_the_other_models(pkg):
    """lum_want_logits is not tied to one family: a Llama-shaped model's rows, and its per-token steps, equal its last-row logits."""
    with pkg.B200Runtime.initialize(device=0) as r:
        r.load_model(pkg.CONFIGS["small_q8"])
        r.synth(3)
        toks = [int(t) for t in np.random.default_rng(1).integers(0, 2048, 40)]
        r.want_logits([0, 7, 39]); r.set_data(toks); r.execute({"s": 40, "p": 0})
        got, last = r.get_wanted(), r.get_f32()
        scale = np.abs(last).max()
        assert np.abs(got[2] - last).max() < 1e-4 * scale
        for row, n in ((0, 1), (1, 8)):
            r.kv_reset(); r.set_data(toks[:n]); r.execute({"s": n, "p": 0})
            assert np.abs(got[row] - r.get_f32()).max() < 5e-3 * scale
        r.kv_reset(); r.want_logits([1]); r.set_data(toks[:3]); r.execute({"s": 3, "p": 0})
        one = r.get_wanted()[0]
        r.kv_reset(); r.set_data(toks[:2]); r.execute({"s": 2, "p": 0})
        assert np.abs(one - r.get_f32()).max() < 1e-5 * scale


# ---- the tools
@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run(pkg, tmp_path, dtype):
    cfg = mc.MIXED
    W = mc.weights(cfg, 90)
    folder = mc.save(pkg, tmp_path / "m", cfg, W)
    out = tmp_path / "out"
    out.mkdir()
    toks = mc.tokens(cfg, 90, 91)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:80], "want": [79, 3]}], "end": []}, {"step": 1, "entries": [{"id": "x", "tokens": toks[80:88], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[88:], "want": [0, 1]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "90"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = mp.forward(cfg, W, toks)
    assert not (out / "1.f32").exists()
    check(np.fromfile(out / "0.f32", "<f4").reshape(2, -1), want[[79, 3]], dtype)
    check(np.fromfile(out / "2.f32", "<f4").reshape(2, -1), want[[88, 89]], dtype)


def test_generate_tool(pkg, tmp_path):
    cfg = mc.MIXED
    W = mc.weights(cfg, 70)
    folder = mc.save(pkg, tmp_path / "m", cfg, W)
    prompts = [mc.tokens(cfg, n, 71 + n) for n in (20, 3)]
    cmd = [sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", folder, "--dtype", "float32", "--max-new", "6", "--max-seq", "128"]
    for p in prompts:
        cmd += ["--prompt", ",".join(map(str, p))]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    for line, p in zip(r.stdout.splitlines(), prompts):
        assert json.loads(line) == {"prompt": p, "tokens": greedy(cfg, W, p, 6)[0]}
