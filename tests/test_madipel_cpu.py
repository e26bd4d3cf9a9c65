"""Madipel without a GPU: the registry's reading of a configuration, checkpoint labels, the trace replay's bookkeeping, and hand checks of
the plain implementation the GPU tests compare with."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import madipel_cases as mc
import madipel_plain as mp

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_configuration_becomes_descriptors(pkg, tmp_path):
    cfg = mc.MIXED
    spec = pkg.models.from_config(cfg, dtype="float32", max_seq=128, max_batch=3)
    d = spec.desc
    assert (d.n_layers, d.hidden, d.vocab, d.max_seq, d.max_batch) == (4, 88, 203, 128, 3)
    assert d.weight_dtype == d.kv_dtype == d.embed_dtype == pkg.DTYPE["f32"]
    assert (round(d.residual_mult, 6), round(d.logit_scale, 6), round(d.rms_eps, 9)) == (0.63, 0.37, 1e-5)
    assert [(g.n_q_heads, g.n_kv_heads, g.qk_dim, g.v_dim, g.window, g.v_mix, g.ffn) for g in spec.layers] == [
        (6, 2, 40, 24, 50, 0, 100), (4, 4, 24, 12, 7, 1, 0), (10, 1, 64, 48, 130, 1, 72), (2, 2, 33, 24, 0, 1, 33)]
    assert abs(spec.layers[2].scale - 0.2) < 1e-7 and abs(spec.layers[0].scale - 40 ** -0.5) < 1e-7
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    assert pkg.models.from_config(str(tmp_path)).desc.kv_dtype == pkg.DTYPE["bf16"]


@pytest.mark.parametrize("change", [dict(architecture="Unknown"), dict(width=0), dict(layers=[]),
                                    dict(layers=[{**mc.layer(4, 2, 16, 16, 8, 32), "type": "recurrent"}]), dict(layers=[mc.layer(5, 2, 16, 16, 8, 32)]),
                                    dict(layers=[{**mc.layer(4, 2, 16, 16, 8, 32), "mlp": {"kind": "routed", "ff": 8}}])])
def test_what_the_design_does_not_have_is_refused(pkg, change):
    with pytest.raises(ValueError):
        pkg.models.from_config({**mc.MIXED, **change})


def test_checkpoint_labels_match_the_weights(pkg, tmp_path):
    for cfg in (mc.MIXED, mc.WIDE):
        W = mc.weights(cfg, 1)
        folder = mc.save(pkg, tmp_path / str(cfg["width"]), cfg, W)
        got, _ = pkg.safetensors_read(os.path.join(folder, "model.safetensors"))
        assert sorted(got) == sorted(pkg.models.from_config(folder).tensor_names())
        assert got["l1.mix.vmix"][1].shape == ()


def test_every_layer_can_have_its_own_sizes(pkg):
    spec = pkg.models.from_config(mc.MIXED)
    n = spec.weight_elems_per_token()
    assert n == sum(v.size for k, v in mc.weights(mc.MIXED, 0).items() if k.split(".")[-1] in ("q", "k", "v", "o", "up", "down", "head"))


def test_tools_answer_without_a_gpu():
    for tool in ("trace_run", "generate"):
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", tool), "--help"], capture_output=True, text=True)
        assert r.returncode == 0 and "--model" in r.stdout
        assert os.access(os.path.join(ROOT, "bin", tool), os.X_OK)


class FakeRuntime:
    """Keeps what the replay asks for; logits of a row = (slot, position, token)."""

    def __init__(self):
        self.calls, self.want, self.released = [], [], []

    def seq_select(self, s): self.slot = s
    def want_logits(self, rows): self.want = list(rows)
    def set_data(self, t): self.tokens = list(t)
    def kv_release(self, s): self.released.append(s)
    def synchronize(self): pass

    def execute(self, dims):
        assert dims["s"] == len(self.tokens)
        self.calls.append((self.slot, dims["p"], len(self.tokens)))
        self.got = [(self.slot, dims["p"] + w, self.tokens[w]) for w in self.want]

    def get_wanted(self): return self.got


def test_trace_replay_keeps_positions_and_slots(pkg):
    rt = FakeRuntime()
    r = pkg.replay.TraceReplay(rt, 2)
    assert r.step([{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], []) == [(0, 2, 7), (0, 0, 5)]      # in the order asked for
    assert r.step([{"id": "b", "tokens": [9], "want": []}], []) == []
    assert r.step([{"id": "a", "tokens": [8], "want": [0, 0]}, {"id": "b", "tokens": [1, 2], "want": [1]}], ["a"]) == [(0, 3, 8), (0, 3, 8), (1, 2, 2)]
    assert rt.released == [0]
    assert r.step([{"id": "a", "tokens": [4], "want": [0]}], ["a", "b"]) == [(0, 0, 4)]                  # a new request in a slot used before
    assert rt.calls == [(0, 0, 3), (1, 0, 1), (0, 3, 1), (1, 1, 2), (0, 0, 1)]
    with pytest.raises(RuntimeError):
        r.step([{"id": i, "tokens": [1], "want": []} for i in "xyz"], [])
    cap = pkg.replay.TraceReplay.capacity(130, 4)
    assert cap["max_seq"] == 192 and cap["kv_pool_pages"] == 3 + 4 and cap["max_batch"] == 4


# ---- the plain implementation, by hand
def test_plain_norms_and_activation():
    x = np.array([[1.0, 2.0, 6.0]])
    assert np.allclose(mp.layer_norm(x, np.array([1.0, 2.0, 3.0]), np.array([0.0, 1.0, -1.0]), 0.5), [[-2 / np.sqrt(14 / 3 + 0.5), 1 - 2 / np.sqrt(14 / 3 + 0.5), 9 / np.sqrt(14 / 3 + 0.5) - 1]])
    assert np.allclose(mp.rms_norm(x, np.ones(3), 0.25), x / np.sqrt(41 / 3 + 0.25))
    sp, sq = np.log(1 + np.exp(0.3)), np.log(1 + np.exp(-0.7))
    z = np.array([2.0, 0.0, -1.5])
    assert np.allclose(mp.xielu(z, 0.3, -0.7), [4 * sp + 1, 0.0, (0.5 + sq) * (np.exp(-1.5) - 1 + 1.5) - 0.75])


def test_plain_positions_window_and_bias():
    s = mp.sinusoid([0, 3], 5)
    assert np.allclose(s[0], [0, 1, 0, 1, 0]) and np.allclose(s[1, 2:4], [np.sin(3 * 10000 ** -0.4), np.cos(3 * 10000 ** -0.4)])
    assert mp.window_mask(4, 2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False], [False, False, True, True]]
    assert np.allclose(mp.distance_bias(3, np.array([2.0]), np.array([0.5]))[0, 2], [2 * np.log(2.0), 2 * np.log(1.5), 0.0])


def test_plain_attention_shares_heads_in_groups():
    # 4 query heads over 2 K/V heads, window 1: every head returns its K/V head's own value
    q, k, v = np.ones((3, 4 * 2)), np.ones((3, 2 * 2)), np.arange(3 * 2 * 2, dtype=float).reshape(3, 4)
    out = mp.attention(q, k, v, 4, 2, 1.0, np.ones(4), np.zeros(4), np.zeros(4), 1)
    assert np.allclose(out.reshape(3, 4, 2), np.stack([v[:, :2], v[:, :2], v[:, 2:], v[:, 2:]], 1))


def test_a_window_one_token_off_shows_in_the_test_models():
    """The tolerance of the GPU tests is far below what a key too many or too few would cause."""
    cfg = mc.config([mc.layer(4, 2, 32, 32, 20, 48)], width=64)
    W, toks = mc.weights(cfg, 3, sharp=3.0), mc.tokens(cfg, 90, 4)
    want = mp.forward(cfg, W, toks)
    for size in (19, 21):
        off = mp.forward(mc.config([mc.layer(4, 2, 32, 32, size, 48)], width=64), W, toks)
        e = mc.errors(off, want)
        assert e[19:].max() > 0.05 and np.median(e[21:]) > 20 * mc.TOL["float32"]
