"""The Fuposun design through the engine: prompts, portions, decode steps, batches and the command line, against the plain
statement in oracle/fuposun_ref.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import fuposun_ref as ur
from oracle.finuvik_ref import save_model
from tests import fuposun_models as fm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
MODELS = {"odd": (fm.ODD, 11), "even": (fm.EVEN, 12)}
EXTRA = {"ones": (fm.ONES, 13)}
TOL = {"f32": 1e-4, "bf16": 4e-2}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, (cfg, seed) in {**MODELS, **EXTRA}.items():
        d = tmp_path_factory.mktemp(name)
        w = fm.weights(cfg, seed)
        save_model(d, cfg, w)
        out[name] = (str(d), cfg, w)
    return out


def open_model(ob, folders, name, kind, max_batch=1, **kw):
    m = ob.open_model(folders[name][0], ob.F32 if kind == "f32" else ob.BF16, max_batch, **kw)
    assert m.design == "Fuposun"
    return m


def err(got, ref):
    """root mean square over the vocabulary of the difference, in units of the spread of the logits; per position"""
    d = np.asarray(got, np.float64) - ref
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / ref.std()


def truth(cfg, w, ids):
    """Logits of every token, and how close its choices of experts were."""
    m = ur.FuposunRef(cfg, w)
    return m.forward(ids), m.margins[0]


def close(got, ref, kind, margins):
    """Every position in float32.  In bfloat16 a token whose choice of experts is a close call may take the other one, which
    also reaches the tokens that look at it (`margins`: how close its own choices were), and a sequence's first tokens are
    touchy: the norm behind the recurrence keeps little more than the sign of their one score."""
    e = err(got, ref)
    if kind == "f32":
        return e.max() < TOL[kind]
    sure = e[np.asarray(margins) > 0.1]
    if len(sure) <= 8:
        return len(sure) == 0 or np.median(sure) < 0.1
    return np.quantile(sure, 0.8) < TOL[kind] and np.median(sure) < TOL[kind] / 2


def whole(m, ids, rows=None):
    rows = list(range(len(ids))) if rows is None else rows
    m.want_logits(rows)
    m.prefill(np.asarray(ids, np.int32)[None])
    return m.row_logits(len(rows))


def prompt(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_whole_prompts(cuda, ob, folders, name, kind):
    _, cfg, w = folders[name]
    m = open_model(ob, folders, name, kind)
    for n in (1, 2, 63, 64, 65, 200):
        ids = prompt(cfg, n, n)
        ref, margins = truth(cfg, w, ids)
        assert close(whole(m, ids), ref, kind, margins), n
    # far beyond every window
    ids = prompt(cfg, 700, 9)
    ref, margins = truth(cfg, w, ids)
    assert close(whole(m, ids), ref, kind, margins)
    m.close()


def test_sizes_and_constants_of_one(cuda, ob, folders):
    _, cfg, w = folders["ones"]
    ids = prompt(cfg, 90, 4)
    ref, _ = truth(cfg, w, ids)
    m = open_model(ob, folders, "ones", "f32")
    assert close(whole(m, ids), ref, "f32", None)
    got = [whole(m, ids[:70])]
    for t in range(70, 90):
        m.decode_step(in_ids=ids[t:t + 1])
        got.append(m.logits(1))
    assert close(np.concatenate(got), ref, "f32", None)
    m.close()
    m = open_model(ob, folders, "ones", "bf16")  # touchy sizes: the kernels take them, and the numbers are numbers
    assert np.isfinite(whole(m, ids)).all() and np.median(err(whole(m, ids), ref)) < 0.3
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_portions_of_any_size(cuda, ob, folders, name, kind):
    _, cfg, w = folders[name]
    ids = prompt(cfg, 150, 3)
    ref, margins = truth(cfg, w, ids)
    m = open_model(ob, folders, name, kind)
    for sizes in ([2] * 75, [1, 2, 3, 58, 2, 64, 20], [64, 64, 22], [149, 1], [31, 33, 1, 1, 84]):
        got, at = [], 0
        for n in sizes:
            part = ids[at:at + n]
            if at and n == 1:
                m.decode_step(in_ids=part)
                got.append(m.logits(1))
            else:
                m.want_logits(range(n))
                (m.extend if at else m.prefill)(part[None])
                got.append(m.row_logits(n))
            at += n
        assert at == len(ids) and close(np.concatenate(got), ref, kind, margins), sizes
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_decoding_token_by_token_is_the_prefill(cuda, ob, folders, name, kind):
    _, cfg, w = folders[name]
    ids = prompt(cfg, 290, 4)  # crosses a row bucket of the captured step
    ref, margins = truth(cfg, w, ids)
    m = open_model(ob, folders, name, kind)
    pre = whole(m, ids)
    for graphs in (True, False):
        m.set_graphs(graphs)
        got = [whole(m, ids[:1])]
        for t in range(1, len(ids)):
            m.decode_step(in_ids=ids[t:t + 1])
            got.append(m.logits(1))
        got = np.concatenate(got)
        assert close(got, ref, kind, margins)
        assert close(got, pre.astype(np.float64), kind, margins)
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_a_batch_is_every_sequence_alone(cuda, ob, folders, name, kind):
    _, cfg, w = folders[name]
    lens = [5, 130, 1, 64, 17]
    prompts = [prompt(cfg, n, 20 + n) for n in lens]
    m = open_model(ob, folders, name, kind, max_batch=5)
    m.prefill_ragged(prompts)
    refs = [ur.FuposunRef(cfg, w) for _ in lens]
    ref = np.stack([r.forward(p)[-1] for r, p in zip(refs, prompts)])
    last = lambda: [r.margins[-1][-1] for r in refs]
    assert close(m.logits(5), ref, kind, last())
    rng = np.random.default_rng(6)
    for step in range(6):
        nxt = rng.integers(0, cfg["vocab"], 5).astype(np.int32)
        if step == 3:  # a further turn of several tokens in between
            more = rng.integers(0, cfg["vocab"], (5, 9)).astype(np.int32)
            m.extend(more)
            ref = np.stack([r.forward(t)[-1] for r, t in zip(refs, more)])
        else:
            m.decode_step(in_ids=nxt)
            ref = np.stack([r.forward([t])[-1] for r, t in zip(refs, nxt)])
        assert close(m.logits(5), ref, kind, last()), step
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_large_batches_take_other_projection_kernels(cuda, ob, folders, kind):
    _, cfg, w = folders["even"]
    B = 40  # beyond the smallest weight-streaming tiles; the same prompt in every other row
    p = [prompt(cfg, 12 + b % 3, 50 + b % 4) for b in range(B)]
    m = open_model(ob, folders, "even", kind, max_batch=B, max_seq_len=64)
    m.prefill_ragged(p)
    refs = {}
    nxt = (np.arange(B) % 7).astype(np.int32)
    m.decode_step(in_ids=nxt)
    got = m.logits(B)
    for b in range(0, B, 9):
        r = ur.FuposunRef(cfg, w)
        r.forward(p[b])
        refs[b] = r.forward([nxt[b]])[-1], r.margins[-1][0]
    ref, margins = (np.stack(x) for x in zip(*refs.values()))
    assert close(got[list(refs)], ref, kind, margins)
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_a_sequence_leaves_nothing_behind(cuda, ob, folders, kind):
    _, cfg, w = folders["odd"]
    a, b = prompt(cfg, 180, 1), prompt(cfg, 33, 2)
    fresh = open_model(ob, folders, "odd", kind)
    want = whole(fresh, b)
    fresh.close()
    m = open_model(ob, folders, "odd", kind)
    whole(m, a)
    for t in range(5):
        m.decode_step(in_ids=a[t:t + 1])
    assert np.array_equal(whole(m, b), want)
    whole(m, a)
    assert np.array_equal(whole(m, b), want)
    m.close()


def test_the_unfused_kernels_agree(cuda, ob, folders):
    _, cfg, w = folders["even"]
    ids = prompt(cfg, 140, 8)
    ref, margins = truth(cfg, w, ids)
    m = open_model(ob, folders, "even", "bf16")
    m.set_prefill_by_decode(2)
    got = [whole(m, ids[:130])]
    for t in range(130, 140):
        m.decode_step(in_ids=ids[t:t + 1])
        got.append(m.logits(1))
    assert close(np.concatenate(got), ref, "bf16", margins)
    m.set_prefill_by_decode(1)  # position by position through the decode kernels
    m.prefill(ids[None])
    assert close(m.logits(1), ref[-1:], "bf16", margins[-1:])
    m.close()


@pytest.mark.parametrize("name", ["odd", "even"])
def test_a_window_passes_over_decoded_tokens(cuda, ob, folders, name):
    """Nothing that left every window and every state's reach may matter: a prompt's first tokens are exchanged, and a model
    of attention layers alone must answer the same once they are out of sight, but not before."""
    cfg = fm.config([l for l in ((fm.attention(window=6), fm.moe()), (fm.attention(heads=2, window=11), None))])
    w = fm.weights(cfg, 5)
    folder = os.path.join(folders[name][0], "windows")
    save_model(folder, cfg, w)
    a = prompt(cfg, 60, 1)
    b = a.copy()
    b[:4] = (b[:4] + 1) % cfg["vocab"]
    reach = 5 + 10  # the last position that the fourth token still touches is 3 + 15
    m = ob.open_model(folder, ob.F32 if name == "odd" else ob.BF16)
    got = []
    for ids in (a, b):
        rows = [whole(m, ids[:10])]
        for t in range(10, 60):
            m.decode_step(in_ids=ids[t:t + 1])
            rows.append(m.logits(1))
        got.append(np.concatenate(rows))
    m.close()
    same = np.abs(got[0] - got[1]).max(-1)
    assert same[3 + reach] > 1e-3 and same[3 + reach + 1:].max() == 0.0


@pytest.mark.parametrize("name", list(MODELS))
def test_greedy_generation(cuda, ob, folders, name):
    """The engine's own loop in float32 takes the plain statement's best token at every step."""
    from onellm_b200.generate import generate
    _, cfg, w = folders[name]
    prompts = [prompt(cfg, n, 70 + n) for n in (40, 7, 23)]
    m = open_model(ob, folders, name, "f32", max_batch=3)
    out = generate(m, prompts, 20)
    for p, row in zip(prompts, out):
        r = ur.FuposunRef(cfg, w)
        lg = r.forward(p)[-1]
        for t in row:
            # the token is the best one, up to a tie within rounding
            assert lg[t] > lg.max() - 1e-3 * lg.std()
            lg = r.forward([t])[-1]
    same = open_model(ob, folders, name, "f32", max_batch=1).generate(prompts[0][None], 20)
    assert np.array_equal(same[0], out[0])
    m.close()


def test_sampling_keeps_to_the_top_k(cuda, ob, folders):
    _, cfg, w = folders["even"]
    ids = prompt(cfg, 9, 31)
    m = open_model(ob, folders, "even", "bf16")
    m.set_sampling(top_k=5, temperature=0.8)
    tok = m.prefill(ids[None])[0]
    assert tok in np.argsort(m.logits(1)[0])[-5:]
    m.close()


def test_positions_beyond_the_model_are_refused(cuda, ob, folders):
    _, cfg, _ = folders["odd"]
    m = open_model(ob, folders, "odd", "bf16", max_seq_len=50)
    assert m.limits() == (cfg["vocab"], 50, 1)
    m.prefill(prompt(cfg, 49, 0)[None])
    m.decode_step(in_ids=np.zeros(1, np.int32))
    with pytest.raises(ob.OnellmError):
        m.decode_step(in_ids=np.zeros(1, np.int32))
    with pytest.raises(ob.OnellmError):
        m.extend(np.zeros((1, 2), np.int32))
    with pytest.raises(ob.OnellmError):
        m.prefill(np.full((1, 3), cfg["vocab"], np.int32))
    m.close()


def test_missing_and_misshapen_tensors_are_refused(cuda, ob, tmp_path):
    w = fm.weights(fm.ODD, 1)
    for change, text in ((lambda x: x.pop("l1.mix.a2.b"), "l1.mix.a2.b"), (lambda x: x.pop("l3.mix.a1"), "l3.mix.a1"),
                         (lambda x: x.pop("l0.mlp.e6.down"), "l0.mlp.e6.down"),
                         (lambda x: x.update({"l0.mix.uk": x["l0.mix.uk"][:-1]}), "l0.mix.uk")):
        x = dict(w)
        change(x)
        save_model(tmp_path, fm.ODD, x)
        with pytest.raises(ob.OnellmError) as e:
            ob.open_model(tmp_path)
        assert e.value.status == -5 and text in str(e.value)


@pytest.mark.parametrize("dtype,kind", [("float32", "f32"), ("bfloat16", "bf16")])
def test_trace_run_program(cuda, ob, folders, tmp_path, dtype, kind):
    folder, cfg, w = folders["odd"]
    a, b = prompt(cfg, 60, 41).tolist(), prompt(cfg, 21, 42).tolist()
    steps, want = [], []
    ra, rb = (truth(cfg, w, x) for x in (a, b))
    for n, (name, lo, hi, rows) in enumerate([("a", 0, 40, [39, 0]), ("a", 40, 41, [0]), ("a", 41, 43, [0, 1]), ("a", 43, 60, []),
                                              ("b", 0, 1, [0]), ("b", 1, 21, [19, 5])]):
        ids, ref = (a, ra) if name == "a" else (b, rb)
        last = hi == len(ids)
        steps.append({"step": n, "entries": [{"id": name, "tokens": ids[lo:hi], "want": rows}], "end": [name] if last else []})
        want.append([x[[lo + r for r in rows]] for x in ref])
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "60"],
                       input="\n".join(json.dumps(s) for s in steps), text=True, capture_output=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert p.stdout.split("\n")[:-1] == [f"done {n}" for n in range(len(steps))]
    for n, (ref, margins) in enumerate(want):
        path = tmp_path / f"{n}.f32"
        if len(ref) == 0:
            assert not path.exists()
            continue
        assert close(np.fromfile(path, "<f4").reshape(ref.shape), ref, kind, margins), n


def test_generate_command(cuda, ob, folders):
    folder, cfg, w = folders["even"]
    p = subprocess.run([sys.executable, "-m", "onellm_b200.generate", "--model", folder, "--dtype", "float32", "--prompt", "3,1,4", "--prompt",
                        "1,5,9,2,6", "--new", "4"], text=True, capture_output=True, cwd=ROOT, timeout=300)
    assert p.returncode == 0, p.stderr
    rows = [[int(x) for x in line.split(",")] for line in p.stdout.split()]
    m = open_model(ob, folders, "even", "f32")
    assert rows[0] == m.generate(np.array([[3, 1, 4]], np.int32), 4)[0].tolist()
    assert rows[1] == m.generate(np.array([[1, 5, 9, 2, 6]], np.int32), 4)[0].tolist()
    m.close()
