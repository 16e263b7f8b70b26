"""No device needed: the Fafelix reader in the model registry (a checkpoint directory opens on the host), refused
configurations, and the oracle's own rules on hand-worked cases."""
import math

import numpy as np
import pytest

import fafelix_oracle as O
from yalm_b200 import api


def three_layers(**kw):
    return O.make_config([O.delta_mixer(), O.attention_mixer(), dict(O.wkv_mixer(), mlp=None)], width=40, vocab=50, ff=56, **kw)


def test_directory_checkpoint_opens_through_the_registry(tmp_path):
    cfg = three_layers(loop=(0, 2, 3))
    folder = str(tmp_path / "m")
    O.write_checkpoint(folder, cfg, O.make_weights(cfg, 1))
    m = api.Model(folder, 0, api.F32)
    assert m.is_stack() and (m.dim, m.vocab_size, m.n_layers) == (40, 50, 3)
    assert (m.n_experts, m.hidden_dim, m.weight_dtype) == (0, 56, api.F32)
    m.close()
    m = api.Model(folder, 100)
    assert m.weight_dtype == api.BF16 and m.max_seq_len == 100      # no table bounds the context: the caller's is taken
    m.close()


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0].update(type="gla"), "a layer type of another design"),
    (lambda c: c.update(width=0), "no width"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "value heads that do not divide over the key heads"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "a convolution without taps"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "query heads that do not divide over the key heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "odd rotated size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "more rotated channels than a head has"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling without a factor"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "scaling bounds in the wrong order"),
    (lambda c: c["layers"][2]["mixer"].update(dim=0), "no head size"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "unknown feed-forward kind"),
    (lambda c: c["layers"][1]["mlp"].update(ff=0), "no hidden size"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "a bigram table without rows"),
    (lambda c: c.update(loop={"start": 1, "stop": 4, "times": 2}), "a span past the last layer"),
    (lambda c: c.update(loop={"start": 2, "stop": 2, "times": 2}), "an empty span"),
    (lambda c: c.update(loop={"start": 0, "stop": 2, "times": 0}), "no passes"),
])
def test_bad_configurations_are_refused(tmp_path, edit, what):
    cfg = three_layers()
    W = O.make_weights(cfg, 2)
    edit(cfg)
    folder = str(tmp_path / "m")
    O.write_checkpoint(folder, cfg, W)
    with pytest.raises(api.YalmError) as e:
        api.Model(folder)
    assert e.value.code == -3, what


def test_interleaved_rotation_on_worked_cases():
    f = O.rotary_freqs({"dims": 4, "base": 100.0})
    assert f.tolist() == [1.0, 0.1]
    x = np.array([1.0, 0.0, 0.0, 2.0, 7.0])                       # pairs (0, 1) and (2, 3); the fifth channel passes unchanged
    np.testing.assert_allclose(O.rotate_pairs(x, 3, f), [math.cos(3.0), math.sin(3.0), -2 * math.sin(0.3), 2 * math.cos(0.3), 7.0], atol=1e-12)
    np.testing.assert_allclose(O.rotate_pairs(x, 0, f), x)


def test_frequencies_by_wavelength():
    rot = {"dims": 8, "base": 300.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}}
    f0, f = O.rotary_freqs({"dims": 8, "base": 300.0}), O.rotary_freqs(rot)
    wave = 2 * math.pi / f0
    assert wave[0] < 64 / 3 and 64 / 3 < wave[1] < 64 and wave[2] > 64          # kept, between, divided
    s = (64 / wave[1] - 1.0) / 2.0
    np.testing.assert_allclose(f, [f0[0], (1 - s) * f0[1] / 4 + s * f0[1], f0[2] / 4, f0[3] / 4])


def test_bigram_rows():
    big = {"buckets": 53, "mul_prev": 31, "mul_cur": 5}
    assert O.bigram_row(None, 7, big) == 53
    assert O.bigram_row(0, 0, big) == 0
    assert O.bigram_row(10, 3, big) == (310 + 15) % 53
    assert O.bigram_row(3, 10, big) != O.bigram_row(10, 3, big)


def test_order_of_layers():
    cfg = {"layers": [None] * 4, "loop": {"start": 1, "stop": 3, "times": 3}}
    assert O.layer_runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert O.layer_runs({"layers": [None] * 2}) == [(0, False), (1, False)]
    assert O.layer_runs({"layers": [None] * 2, "loop": {"start": 0, "stop": 1, "times": 2}}) == [(0, False), (0, True), (1, False)]


def test_recurrences_on_worked_cases():
    one = np.ones((3, 1))
    # delta rule, one channel: the write replaces what the (decayed) state holds for the key by the share beta of the new value
    out = O.delta_rule(one, one, np.array([[2.0], [4.0], [0.0]]), np.array([0.5, 0.5, 1.0]), np.array([1.0, 0.5, 0.0]))
    np.testing.assert_allclose(out[:, 0], [2.0, 1.0 + 0.5 * (4.0 - 1.0), 2.5])
    # time mixing: the current token counts with the bonus, earlier ones with the decays of the tokens after them (not their own)
    out = O.wkv_rule(one, np.array([[1.0], [2.0], [3.0]]), np.array([[1.0], [1.0], [1.0]]), np.array([[0.5], [0.1], [0.9]]), np.array([10.0]))
    np.testing.assert_allclose(out[:, 0], [10.0, 1.0 + 20.0, 0.1 * 1.0 + 2.0 + 30.0])
    c = O.short_conv(np.array([[1.0], [2.0], [4.0]]), np.array([[3.0, 10.0]]))     # the last tap is the current position's
    np.testing.assert_allclose(c[:, 0], [10.0, 23.0, 46.0])


def test_sink():
    s = np.array([0.0, math.log(2.0)])
    np.testing.assert_allclose(O.softmax_with_sink(s, math.log(3.0)), [1 / 6, 2 / 6])      # the sink takes its share and gives nothing back
    np.testing.assert_allclose(O.softmax_with_sink(s + 1000.0, 0.0), [1 / 3, 2 / 3])
    np.testing.assert_allclose(O.softmax_with_sink(s, 1000.0), [0.0, 0.0], atol=1e-300)
