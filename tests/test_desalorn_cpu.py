"""No device needed: the Desalorn reader in the model registry (a checkpoint directory opens on the host), refused configurations, and
the oracle's own rules on hand-worked cases."""
import math

import numpy as np
import pytest

import desalorn_oracle as O
from yalm_b200 import api


def three_layers(**kw):
    return O.make_config([("attention", O.attention_mixer(), O.moe_mlp()), ("retention", O.retention_mixer(), None), ("latent_attention", O.latent_mixer(), O.moe_mlp(ff=28))],
                         width=42, vocab=50, **kw)


def test_directory_checkpoint_opens_through_the_registry(tmp_path):
    cfg = three_layers()
    folder = str(tmp_path / "m")
    O.write_checkpoint(folder, cfg, O.make_weights(cfg, 1))
    m = api.Model(folder, 0, api.F32)
    assert m.is_stack() and (m.dim, m.vocab_size, m.n_layers) == (42, 50, 3)
    assert (m.n_experts, m.hidden_dim, m.weight_dtype) == (6, 40, api.F32)
    m.close()
    m = api.Model(folder, 100)
    assert m.weight_dtype == api.BF16 and m.max_seq_len == 100      # no table bounds the context: the caller's is taken
    m.close()


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0].update(type="wkv"), "a layer type of another design"),
    (lambda c: c.update(width=0), "no width"),
    (lambda c: c["norm"].update(groups=4), "norm groups that do not divide the width"),
    (lambda c: c["norm"].update(groups=0), "no norm group"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "query heads that do not divide over the key heads"),
    (lambda c: c["layers"][0]["mixer"].update(bias_max=0), "no farthest distance"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "a negative cap"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decays that are not one per head"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "odd rotated size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "more rotated channels than a head has"),
    (lambda c: c["layers"][2]["mixer"].update(q_rank=0), "no query latent"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=18), "more rotated channels than the key part has"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(ff=0), "no hidden size"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups that do not divide the experts"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "more groups kept than there are"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "more experts chosen than the kept groups have"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "a shared expert without a hidden size"),
])
def test_refused_configurations(tmp_path, edit, what):
    cfg = three_layers()
    W = O.make_weights(cfg, 1)
    edit(cfg)
    folder = str(tmp_path / "m")
    O.write_checkpoint(folder, cfg, W)
    with pytest.raises(api.YalmError):
        api.Model(folder, 0, api.F32)


def test_distance_buckets():
    rows, far = 16, 128                                             # exact below 8, then eight rows up to 128: a factor sqrt(2) each
    assert [O.bucket(n, rows, far) for n in range(8)] == list(range(8))
    assert [O.bucket(n, rows, far) for n in (8, 11, 12, 15, 23, 127, 128, 5000)] == [8, 8, 9, 9, 11, 15, 15, 15]


def test_group_norm_by_hand():
    x = np.array([3.0, 4.0, 0.0, 10.0])
    got = O.group_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), 2, 0.5)
    np.testing.assert_allclose(got, [3 / math.sqrt(13), 8 / math.sqrt(13), 0.0, 10 / math.sqrt(50.5)])


def test_choice_over_groups():
    choice = np.array([-0.1, -9.0, -1.0, -1.1, -0.9, -5.0])          # pairs: -9.1, -2.1, -5.9
    assert O.choose(choice, 2, 3, 1).tolist() == [2, 3]
    assert O.choose(choice, 2, 3, 2).tolist() == [4, 2]
    assert O.choose(choice, 2, 3, 3).tolist() == [0, 4]


def test_retention_by_hand():
    q = np.ones((3, 1, 1))
    k, v = np.array([[[1.0]], [[2.0]], [[0.0]]]), np.array([[[1.0]], [[3.0]], [[9.0]]])
    np.testing.assert_allclose(O.retention_scan(q, k, v, np.array([0.5]))[:, 0, 0], [1.0, 6.5, 3.25])


def test_half_split_and_interleaved_rotation():
    f = np.array([math.pi / 2, 0.0])
    x = np.array([1.0, 2.0, 3.0, 4.0, 5.0])
    np.testing.assert_allclose(O.rotate(x, 1, f, False), [-3.0, 2.0, 1.0, 4.0, 5.0], atol=1e-12)
    np.testing.assert_allclose(O.rotate(x, 1, f, True), [-2.0, 1.0, 3.0, 4.0, 5.0], atol=1e-12)
