"""The Fuposun design without a GPU: the plain statement against itself and hand-computed values, and what the
configuration reader refuses before it touches a device."""
import copy
import json

import numpy as np
import pytest

from oracle import finuvik_ref as fr
from oracle import fuposun_ref as ur
from tests import fuposun_models as fm


def test_mechanisms_on_hand_computed_values():
    # a window of three: itself and two before
    assert [j for j in range(9) if ur.visible(6, j, 3)] == [4, 5, 6] and [j for j in range(9) if ur.visible(1, j, 3)] == [0, 1]
    # equal scores: the mean of the visible values; one key: its value whatever the score
    c = np.array([[1.0], [2.0], [6.0]])
    one = np.ones((1, 1))
    o = ur.latent_attention(np.zeros((3, 1, 1)), c, one, one, [0, 1, 2], [0, 1, 2], 1.0, 2)
    assert np.allclose(o[:, 0, 0], [1.0, 1.5, 4.0])
    o = ur.latent_attention(np.full((1, 1, 1), 9.0), c, one, 3 * one, [2], [0, 1, 2], 1.0, 1)
    assert np.allclose(o, 18.0)
    # two keys a distance log(3) / scale apart in score
    o = ur.latent_attention(np.ones((1, 1, 1)), np.array([[0.0], [np.log(3.0)]]), one, one, [1], [0, 1], 1.0, 2)
    assert np.isclose(o[0, 0, 0], 0.75 * np.log(3.0))
    assert np.allclose(ur.channel_decay(np.array([0.0, 40.0, -3.0]), 2.0), [0.5 ** 0.5, 1.0, (1 / (1 + np.exp(3.0))) ** 0.5])
    # the decay acts on the rows of key channels; the query reads the new state
    s = np.zeros((1, 2, 1))
    q = np.array([[[1.0, 1.0]], [[1.0, 0.0]]])
    k = np.array([[[2.0, 3.0]], [[0.0, 0.0]]])
    o = ur.gated_linear_attention(q, k, np.ones((2, 1, 1)), np.array([[[0.5, 0.5]], [[0.5, 0.25]]]), s)
    assert np.allclose(o[:, 0, 0], [5.0, 1.0]) and np.allclose(s[0, :, 0], [1.0, 0.75])


def test_experts_on_hand_computed_values():
    # router logits 1, 3, 3: the lower number of equal ones first, scores not renormalised
    h = np.array([[1.0]])
    chosen, w = ur.route(h, np.array([[1.0], [3.0], [3.0]]), 2)
    assert chosen.tolist() == [[1, 2]] and np.allclose(w, 1 / (1 + np.exp(-3.0)))
    # the weight goes into the expert: through a gate that is bounded this is not a factor of its output
    e = (np.array([[4.0]]), np.array([[0.0]]), np.array([[1.0]]))
    y = ur.mixture(h, np.array([[0.0]]), 1, [e], 3.0)
    assert np.isclose(y[0, 0], 2.0 / (1 + np.exp(-3.404)))


@pytest.mark.parametrize("cfg", [fm.ODD, fm.EVEN], ids=["odd", "even"])
def test_portions_do_not_change_the_plain_statement(cfg):
    w = fm.weights(cfg, 1)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    whole = ur.FuposunRef(cfg, w).forward(ids)
    m = ur.FuposunRef(cfg, w)
    parts = np.concatenate([m.forward(ids[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 21), (21, 30))])
    assert np.abs(parts - whole).max() < 1e-9
    assert np.abs(whole).max() < cfg["logit_softcap"]


def _refused(ob, cfg, text, status=-5):
    with pytest.raises(ob.OnellmError) as e:
        ob.Model(cfg)
    assert e.value.status == status and text in str(e.value), str(e.value)


def test_configurations_that_are_refused(ob):
    base = fm.config([(fm.attention(), fm.moe()), (fm.gla(), fm.dense())])

    def changed(fn):
        c = copy.deepcopy(base)
        fn(c)
        return c
    _refused(ob, changed(lambda c: c.pop("residual_mult")), "config.residual_mult")
    _refused(ob, changed(lambda c: c.update(logit_softcap=None)), "config.logit_softcap")
    _refused(ob, changed(lambda c: c["layers"][1].update(type="other")), "layers[1]: unknown type")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"].pop("mask")), "layers[0].mixer.mask")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)), "sizes of layers[0]")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"].pop("q_rank")), "layers[0].mixer.q_rank")
    _refused(ob, changed(lambda c: c["layers"][0]["mlp"].update(kind="other")), "unknown kind")
    _refused(ob, changed(lambda c: c["layers"][0]["mlp"]["router"].update(top=8)), "sizes of layers[0]")
    _refused(ob, changed(lambda c: c["layers"][0]["mlp"].pop("shared")), "layers[0].mlp.shared")
    _refused(ob, changed(lambda c: c["layers"][1]["mixer"].pop("tau")), "layers[1].mixer.tau")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"].update(dim=264)), "above 256", status=-2)


def test_a_folder_without_weights_is_refused(ob, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(fm.ODD))
    with pytest.raises(ob.OnellmError) as e:
        ob.open_model(tmp_path)
    assert e.value.status == -5 and "model.safetensors" in str(e.value)


def test_the_oracle_reads_what_it_wrote(tmp_path):
    w = fm.weights(fm.ODD, 4)
    fr.save_model(tmp_path, fm.ODD, w)
    back = fr.read_safetensors(tmp_path / "model.safetensors")
    assert set(back) == set(w) and all(np.array_equal(back[n], w[n]) for n in w)
