"""Redenex without a GPU: the registry's reading of a configuration, checkpoint labels, the order of layer runs, and hand checks of the plain
implementation the GPU tests compare with."""
import os

import numpy as np
import pytest

import redenex_cases as rc
import redenex_plain as rp


def test_configuration_becomes_descriptors(pkg):
    spec = pkg.models.from_config(rc.MIXED, dtype="float32", max_seq=128, max_batch=3)
    d = spec.desc
    assert (d.block_kind, d.norm_kind, d.n_layers, d.hidden, d.vocab, d.streams, d.max_seq, d.max_batch) == (2, 2, 6, 88, 203, 3, 128, 3)
    assert (d.loop_start, d.loop_stop, d.loop_times) == (1, 3, 3) and abs(d.embed_scale - 0.7) < 1e-7 and abs(d.rms_eps - 1e-5) < 1e-12
    assert d.weight_dtype == d.kv_dtype == d.embed_dtype == pkg.DTYPE["f32"]
    g = spec.layers
    assert [(x.mixer, x.conv_taps, x.ffn) for x in g] == [(1, 3, 100), (0, 4, 70), (1, 2, 0), (0, 1, 0), (0, 5, 72), (0, 4, 33)]
    assert [(x.rec_width, x.rec_blocks) for x in g if x.mixer] == [(84, 7), (40, 1)]
    assert [(x.n_q_heads, x.n_kv_heads, x.qk_dim, x.v_dim, x.chunk, x.rot_dims, x.maps) for x in g if not x.mixer] == [
        (6, 2, 40, 24, 50, 24, 2), (4, 4, 24, 12, 7, 24, 2), (10, 1, 64, 48, 130, 64, 2), (2, 2, 34, 20, 0, 2, 2)]
    assert abs(g[1].ffn_limit - 0.8) < 1e-6 and abs(g[3].diff - 0.6) < 1e-6 and g[4].rot_base == 500.0 and abs(g[4].scale - 0.2) < 1e-7
    plain = pkg.models.from_config({**rc.MIXED, "loop": None}).desc
    assert plain.loop_times == 1


@pytest.mark.parametrize("change", [dict(width=0), dict(layers=[]), dict(streams=0), dict(loop={"start": 2, "stop": 9, "times": 2}),
                                    dict(layers=[{**rc.rec(16, 2, 8), "type": "recurrent"}]), dict(layers=[rc.rec(17, 2, 8)]), dict(layers=[rc.att(5, 2, 16, 16, 8, 32)]),
                                    dict(layers=[rc.att(4, 2, 16, 16, 8, 32, rot=18)]), dict(layers=[{**rc.rec(16, 2, 8), "mlp": {"kind": "routed", "ff": 8}}])])
def test_what_the_design_does_not_have_is_refused(pkg, change):
    with pytest.raises(ValueError):
        pkg.models.from_config({**rc.MIXED, "loop": None, **change})


def test_checkpoint_labels_match_the_weights(pkg, tmp_path):
    for cfg in (rc.MIXED, rc.WIDE):
        W = rc.weights(cfg, 1)
        folder = rc.save(pkg, tmp_path / str(cfg["width"]), cfg, W)
        got, _ = pkg.safetensors_read(os.path.join(folder, "model.safetensors"))
        spec = pkg.models.from_config(folder)
        assert sorted(got) == sorted(spec.tensor_names())
        linear = ("q", "k", "v", "o", "y", "x", "ra", "ri", "gate", "up", "down")
        order = rp.layer_order(len(cfg["layers"]), cfg["loop"])
        assert spec.weight_elems_per_token() == W["head"].size + sum(
            v.size for i in order for k, v in W.items() if k.startswith(f"l{i}.") and k.split(".", 1)[1].replace("mix.", "").replace("mlp.", "") in linear)


def test_order_of_layer_runs(pkg):
    from oneiron_luminal_b200.runtime import layer_order
    for n, loop in ((6, (1, 3, 3)), (4, (0, 4, 2)), (3, (2, 3, 4)), (5, (1, 1, 7)), (2, (0, 1, 1))):
        cfg = rc.config([rc.rec(16, 2, 8)] * n, loop=loop)
        assert layer_order(pkg.models.from_config(cfg).desc, n) == rp.layer_order(n, cfg["loop"])
    assert rp.layer_order(6, dict(start=1, stop=3, times=3)) == [0, 1, 2, 1, 2, 1, 2, 3, 4, 5]


# ---- the plain implementation, by hand
def test_plain_elementwise():
    assert np.allclose(rp.centred_rms_norm(np.array([[3.0, 4.0]]), np.array([0.0, 1.0]), 0.5), [[3 / np.sqrt(13), 8 / np.sqrt(13)]])
    assert np.allclose(rp.softplus(np.array([0.0, 2.0])), [np.log(2), np.log(1 + np.exp(2))])
    z = 1.3
    assert np.allclose(rp.gelu_tanh(z), 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3))))
    assert np.allclose(rp.clamped_gate(np.array([5.0, -9.0]), np.array([-5.0, 5.0]), 2.0), [2 / (1 + np.exp(-3.404)) * -1, -9 / (1 + np.exp(1.702 * 9)) * 3])
    assert np.allclose(rp.short_conv(np.array([[1.0], [2.0], [4.0]]), np.array([[100.0, 10.0, 1.0]])), [[1], [12], [124]])
    assert np.allclose(rp.block_diagonal(np.array([[1.0, 2.0, 3.0, 4.0]]), np.array([[[1, 2], [3, 4]], [[0, 1], [1, 0]]]), np.array([[0, 0], [0.5, 0]])), [[5, 11, 4.5, 3]])


def test_plain_recurrence():
    r, i, lam, u = np.array([[0.5], [1.0]]), np.array([[0.25], [0.5]]), np.array([-1.0]), np.array([[2.0], [3.0]])
    sp = np.log1p(np.exp(-1.0))
    a = np.exp(-8 * r[:, 0] * sp)
    s0 = np.sqrt(1 - a[0] ** 2) * 0.5
    assert np.allclose(rp.gated_recurrence(u, r, i, lam)[:, 0], [s0, a[1] * s0 + np.sqrt(1 - a[1] ** 2) * 1.5])


def test_plain_rotation_chunks_and_difference():
    x = np.arange(1.0, 6.0).reshape(1, 1, 5)
    c, s = np.cos([3, 3 * 0.1]), np.sin([3, 3 * 0.1])
    assert np.allclose(rp.rotate(x, [3], 4, 100.0)[0, 0], [1 * c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + 1 * s[0], 4 * c[1] + 2 * s[1], 5])
    assert rp.chunk_mask(5, 2).astype(int).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    # one visible key: both maps return its value, and the difference is (1 - lambda) v, normed
    v = np.array([[[1.0, 2.0]], [[3.0, -1.0]]])
    q, k = np.ones((2, 2, 2, 3)), np.ones((2, 1, 2, 3))
    o = rp.differential_attention(q, k, v, 2, 1, 1.0, 0.25, 0.5, 1, 0.1)
    one = 0.75 * v[:, 0]
    assert np.allclose(o, np.tile(one / np.sqrt((one ** 2).mean(-1, keepdims=True) + 0.1) * 0.5, 2))
    assert np.allclose(rp.difference_weight(np.array([1.0, 2.0]), np.array([0.5, 0.0]), np.array([1.0, 1.0]), np.array([-1.0, 0.5]), 0.3), np.exp(0.5) - np.exp(-0.5) + 0.3)


def test_plain_streams():
    xs = np.array([[[1.0]], [[10.0]]])
    assert rp.stream_input(xs, np.array([2.0, 0.5])).item() == 7.0
    out = rp.stream_update(xs, np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([100.0, 1000.0]), np.array([[1.0]]))
    assert out[:, 0, 0].tolist() == [1 + 30 + 100, 2 + 40 + 1000]


def test_a_fault_of_one_token_shows_in_the_test_models():
    """A chunk one token longer, a lost state, another order of a loop: far above the tolerance of the GPU tests."""
    W, toks = rc.weights(rc.MIXED, 3, sharp=2.0), rc.tokens(rc.MIXED, 90, 4)
    want = rp.forward(rc.MIXED, W, toks)
    for change in ("size", "loop", "conv"):
        cfg, W2 = {**rc.MIXED, "layers": [dict(l, mixer=dict(l["mixer"])) for l in rc.MIXED["layers"]]}, dict(W)
        if change == "size":
            cfg["layers"][1]["mixer"]["mask"] = {"size": 51}
        elif change == "loop":
            cfg["loop"] = dict(start=1, stop=3, times=2)
        else:
            W2["l0.mix.conv"] = np.roll(W["l0.mix.conv"], 1, axis=1)
        assert rc.errors(rp.forward(cfg, W2, toks), want).max() > 0.05
    assert rc.errors(rp.forward(rc.MIXED, W, toks[1:]), want[1:])[:40].min() > 100 * rc.TOL["float32"]      # the first token is remembered
