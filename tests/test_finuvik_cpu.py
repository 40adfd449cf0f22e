"""The Finuvik design without a GPU: the plain statement against itself and hand-computed values, and what the
configuration reader refuses before it touches a device."""
import copy
import json

import numpy as np
import pytest

from oracle import finuvik_ref as fr
from tests import finuvik_models as fm


def test_mechanisms_on_hand_computed_values():
    assert np.allclose(fr.zero_centred_rms_norm(np.array([[3.0, 4.0]]), np.array([0.0, 1.0]), 0.0), [[3 / 12.5 ** .5, 8 / 12.5 ** .5]])
    # positions 0..2 are in block 0 of 4, position 3 completes it
    assert fr.query_temperature(2, 0.5, 4) == 1.0 and np.isclose(fr.query_temperature(3, 0.5, 4), 1 + 0.5 * np.log(2))
    assert np.isclose(fr.distance_penalty(0, 2.0, 0.3), 0.0) and np.isclose(fr.distance_penalty(10, 2.0, 0.3), 2 * np.log(4))
    # one key: weight one whatever the penalty; two equal keys: the nearer one weighs (1 + r2)^r1 times the other
    v = np.array([[[1.0]], [[0.0]]])
    o = fr.biased_attention(np.ones((2, 1, 1)), np.ones((2, 1, 1)), v, [0, 1], 1.0, [2.0], [1.0], 0.0, 1)
    assert np.allclose(o[:, 0, 0], [1.0, 1 / 5])
    f = fr.forget_gate(np.array([0.0, 50.0, -50.0]), np.array([0.2, 0.2, 0.2]))
    assert np.allclose(f, [0.6, 1.0, 0.2])
    s = np.zeros((1, 1, 1))
    o = fr.gated_recurrence(np.ones((2, 1, 1)), np.full((2, 1, 1), 0.75), np.ones((2, 1, 1)), s)
    assert np.allclose(o[:, 0, 0], [0.25, 0.4375]) and np.isclose(s[0, 0, 0], 0.4375)


@pytest.mark.parametrize("cfg", [fm.ODD, fm.EVEN], ids=["odd", "even"])
def test_portions_do_not_change_the_plain_statement(cfg):
    w = fm.weights(cfg, 1)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    whole = fr.FinuvikRef(cfg, w).forward(ids)
    m = fr.FinuvikRef(cfg, w)
    parts = np.concatenate([m.forward(ids[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 21), (21, 30))])
    assert np.abs(parts - whole).max() < 1e-9


def test_layers_with_shared_weights_keep_memory_of_their_own():
    shared = fm.config([fm.layer(), fm.layer(weights_of=0)])
    twice = fm.config([fm.layer(), fm.layer()])
    w = fm.weights(shared, 3)
    w2 = dict(w, **{n.replace("l0.", "l1."): a for n, a in w.items() if n.startswith("l0.")})
    ids = np.arange(12)
    a, b = fr.FinuvikRef(shared, w).forward(ids), fr.FinuvikRef(twice, w2).forward(ids)
    assert np.array_equal(a, b)


def test_safetensors_round_trip(tmp_path):
    w = fm.weights(fm.ODD, 4)
    fr.save_model(tmp_path, fm.ODD, w)
    back = fr.read_safetensors(tmp_path / "model.safetensors")
    assert set(back) == set(w) and all(np.array_equal(back[n], w[n]) for n in w)
    assert json.load(open(tmp_path / "config.json")) == fm.ODD


def _refused(ob, cfg, text, status=-5):
    with pytest.raises(ob.OnellmError) as e:
        ob.Model(cfg)
    assert e.value.status == status and text in str(e.value), str(e.value)


def test_configurations_that_are_refused(ob):
    base = fm.config([fm.layer(), fm.layer()])

    def changed(fn):
        c = copy.deepcopy(base)
        fn(c)
        return c
    _refused(ob, changed(lambda c: c.pop("architecture")), "architecture")
    _refused(ob, changed(lambda c: c.update(architecture="Nothing")), "unknown architecture")
    _refused(ob, changed(lambda c: c.pop("width")), "config.width")
    _refused(ob, changed(lambda c: c["layers"][1].update(type="other")), "layers[1]: unknown type")
    _refused(ob, changed(lambda c: c["layers"][0]["mlp"].update(kind="experts")), "unknown kind")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"]["left"].pop("vdim")), "layers[0].mixer.left.vdim")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4)), "sizes of layers[0]")
    _refused(ob, changed(lambda c: c["layers"][0]["mixer"]["right"].update(dim=264)), "above 256", status=-2)
    _refused(ob, changed(lambda c: [c["layers"][0].update(weights_of=1), c["layers"][1].update(weights_of=0)]), "circle")
    _refused(ob, changed(lambda c: [c["layers"][1].update(weights_of=0), c["layers"][1]["mlp"].update(ff=80)]), "other sizes")


def test_a_folder_without_the_files_is_refused(ob, tmp_path):
    with pytest.raises(ob.OnellmError) as e:
        ob.open_model(tmp_path)
    assert e.value.status == -5 and "config.json" in str(e.value)
    (tmp_path / "config.json").write_text('{"architecture": "Finuvik", }')
    with pytest.raises(ob.OnellmError) as e:
        ob.open_model(tmp_path)
    assert e.value.status == -5 and "not JSON" in str(e.value)


def test_trace_runner_feeds_prefill_extension_and_decode_steps():
    from onellm_b200.trace_run import TraceRunner

    class Fake:
        def __init__(self):
            self.calls = []

        def set_sampling(self, top_k):
            self.calls.append(("top_k", top_k))

        def want_logits(self, rows):
            self.rows = list(rows)

        def prefill(self, ids):
            self.calls.append(("prefill", ids[0].tolist()))

        def extend(self, ids):
            self.calls.append(("extend", ids[0].tolist()))

        def decode_step(self, in_ids):
            self.calls.append(("decode", in_ids.tolist()))

        def sync(self):
            pass

        def row_logits(self, n):
            return np.array([[r, r] for r in self.rows], np.float32)

        def logits(self, n):
            return np.array([[7, 7]], np.float32)

    m = Fake()
    run = TraceRunner(m)
    assert run.feed("a", [5], []) is None  # a first token is a prefill even when it comes alone
    assert run.feed("a", [6], [0, 0]).tolist() == [[7, 7], [7, 7]]
    assert run.feed("a", [1, 2, 3], [2, 0]).tolist() == [[2, 2], [0, 0]]
    run.end("a")
    assert run.feed("b", [9, 9], [1]).tolist() == [[1, 1]]
    assert m.calls == [("top_k", 0), ("prefill", [5]), ("decode", [6]), ("extend", [1, 2, 3]), ("prefill", [9, 9])]
    with pytest.raises(ValueError):
        run.feed("a", [1], [])


def test_build_knows_the_files_of_every_design():
    from onellm_b200 import build
    have = set(build.sources())
    for name, files in build.DESIGN_SOURCES.items():
        assert set(files) | set(build.ENGINE_SOURCES) <= have, name
