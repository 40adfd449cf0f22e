"""Every mechanism of the Finuvik design alone, against the plain statement in oracle/finuvik_ref.py, in float32 and
bfloat16.  Scores are made to stand out where random ones would hide a misplaced key."""
import numpy as np
import pytest

from oracle import finuvik_ref as fr
from tests.conftest import rel_err
from tests.device import Dev, host, rounded

pytestmark = pytest.mark.gpu
TOL = {"f32": 2e-5, "bf16": 1.2e-2}


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width,ld", [(88, 96), (1024, 1024), (9000, 9008)])
def test_two_zero_centred_norms(cuda, ob, kind, width, ld):
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(0)
    x = np.zeros((5, ld), np.float32)
    x[:, :width] = rng.standard_normal((5, width)) * np.array([1e-3, 1, 30, 1, 0])[:, None]
    w = np.zeros((2, ld), np.float32)
    w[:, :width] = 0.5 * rng.standard_normal((2, width))
    rows = [3, 0, 4, 2]
    o1, o2 = d.zeros(4, ld), d.zeros(4, ld)
    ob.norm_rows(d.dtype, d.f32(x), d.i32(rows), 4, d.f32(w[0]), d.f32(w[1]), o1, o2, 1e-5, width, ld, w_base=1.0)
    for o, wi in ((o1, w[0]), (o2, w[1])):
        ref = fr.zero_centred_rms_norm(x[rows, :width].astype(np.float64), wi[:width], 1e-5)
        assert rel_err(host(o)[:, :width], ref) < TOL[kind]
        assert np.all(host(o)[:, width:] == 0)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("M", [1, 7, 16, 33, 64, 65, 300])
def test_projection_forms(cuda, ob, kind, M):
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(M)
    K, N, ldy = 176, 200, 320
    x, w1, w2 = (rounded(rng.standard_normal(s), kind) for s in ((M, K), (K, N), (K, N)))
    xd, w1d, w2d = d.up(x), d.up(w1), d.up(w2)
    y = d.zeros(M, N)
    ob.project(d.dtype, xd, w1d, None, y, M, N, K)
    assert rel_err(host(y), x @ w1) < TOL[kind]
    # gated, into columns of a wider buffer
    y = d.zeros(M, ldy)
    ob.project(d.dtype, xd, w1d, w2d, y.data_ptr() + 64 * y.element_size(), M, N, K, ldy=ldy, act=ob.GATE_RELU)
    got = host(y)
    assert rel_err(got[:, 64:64 + N], np.maximum(x @ w1, 0) * (x @ w2)) < TOL[kind]
    assert np.all(got[:, :64] == 0) and np.all(got[:, 64 + N:] == 0)
    # added to a float stream in place
    r = rng.standard_normal((M, N)).astype(np.float32) * 50
    rd = d.f32(r)
    ob.project(d.dtype, xd, w1d, None, rd, M, N, K, f32=True, resid=rd)
    assert rel_err(host(rd), x @ w1 + r) < 2e-5  # products of exact inputs, float accumulation and sum


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_embedding_with_positions(cuda, ob, kind):
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(1)
    ld, vocab, n_pos = 48, 30, 40
    tab, pos = rounded(rng.standard_normal((vocab, ld)), kind), rounded(rng.standard_normal((n_pos, ld)), kind)
    td, pd, bad = d.up(tab), d.up(pos), d.i32([0, 0])
    ids = [3, 29, 0, 7, 7, 1]
    out = d.zeros(6, ld, f32=True)
    tp = ob.TokenPositions(d.i32([0, 4, 6]).data_ptr(), d.i32([0, 31]).data_ptr(), 2, None, None)
    ob.embedding_pos(d.dtype, d.i32(ids), out, td, pd, 6, ld, vocab, n_pos, tp, bad)
    assert np.abs(host(out) - (tab[ids] + pos[[0, 1, 2, 3, 31, 32]])).max() < 1e-6
    # decode step: one token per sequence at step - 1 + off
    tp = ob.TokenPositions(None, None, 3, d.i32([40]).data_ptr(), d.i32([0, -5, -39]).data_ptr())
    ob.embedding_pos(d.dtype, d.i32([5, 6, 8]), out, td, pd, 3, ld, vocab, n_pos, tp, bad)
    assert np.abs(host(out)[:3] - (tab[[5, 6, 8]] + pos[[39, 34, 0]])).max() < 1e-6
    assert bad.cpu().tolist() == [0, 0]
    ob.embedding_pos(d.dtype, d.i32([5, 30, 8]), out, td, pd, 3, ld, vocab, 39, tp, bad)
    assert bad.cpu().tolist() == [1, 1]


# ---- attention ---------------------------------------------------------------------------------------------
SIZES = [  # H, G, dk, dv
    (4, 1, 64, 128), (3, 3, 16, 32), (6, 2, 48, 80), (8, 2, 128, 128), (2, 1, 256, 256), (4, 4, 96, 192), (20, 1, 64, 64),
    (2, 2, 128, 16)]


class Attn:
    """A cache of B sequences filled with random keys and values, and the parameters of a launch."""

    def __init__(self, cuda, ob, kind, H, G, dk, dv, lens, S, seed=0, r1=None, coef=0.4, every=16):
        self.ob, self.kind, self.d = ob, kind, Dev(cuda, ob, kind)
        self.H, self.G, self.dk, self.dv, self.S, self.lens = H, G, dk, dv, S, lens
        rng = np.random.default_rng(seed)
        self.rng = rng
        self.k = [rounded(rng.standard_normal((n, G, dk)), kind) for n in lens]
        self.v = [rounded(rng.standard_normal((n, G, dv)), kind) for n in lens]
        self.r1 = np.linspace(0.0, 1.5, H).astype(np.float32) if r1 is None else np.full(H, r1, np.float32)
        self.r2 = np.linspace(0.6, 0.05, H).astype(np.float32)
        self.scale, self.coef, self.every = 1.0 / np.sqrt(dk), coef, every
        d = self.d
        self.qf, self.pen = d.zeros(S, f32=True), d.zeros(H, S, f32=True)
        ob.query_factor(self.qf, S, self.scale, coef, every)
        ob.distance_penalty(self.pen, d.f32(self.r1), d.f32(self.r2), H, S)
        # unused rows hold what a freed sequence may leave behind
        self.kc = d.zeros(len(lens), G, S, dk) + float("nan")
        self.vc = d.zeros(len(lens), G, S, dv) + float("nan")

    def queries(self, counts):
        return [rounded(self.rng.standard_normal((n, self.H, self.dk)), self.kind) for n in counts]

    def params(self, q, k, v, scale_out=1.0):
        """One packed projection buffer [T, q | k | v] and an output with columns around the attention's."""
        T = len(q)
        row = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1)
        self.row = self.d.up(row)
        es = self.row.element_size()
        self.out = self.d.zeros(T, self.H * self.dv + 32)
        p = self.row.data_ptr()
        return self.ob.BiasedAttn(self.d.dtype, self.H, self.G, self.dk, self.dv, p, p + self.H * self.dk * es,
                                  p + (self.H + self.G) * self.dk * es, row.shape[1], self.kc.data_ptr(), self.vc.data_ptr(), self.S,
                                  self.qf.data_ptr(), self.pen.data_ptr(), self.out.data_ptr() + 16 * es, self.H * self.dv + 32, scale_out)

    def result(self):
        o = host(self.out)
        assert np.all(o[:, :16] == 0) and np.all(o[:, -16:] == 0)
        return o[:, 16:-16].reshape(len(o), self.H, self.dv)

    def reference(self, b, q, pos):
        return fr.biased_attention(q, self.k[b], self.v[b], pos, self.scale, self.r1, self.r2, self.coef, self.every)

    def fill(self, upto):
        """The first upto[b] rows of every sequence through the store kernel."""
        counts = [int(n) for n in upto]
        T = sum(counts)
        if T == 0:
            return
        k = np.concatenate([self.k[b][:n] for b, n in enumerate(counts)])
        v = np.concatenate([self.v[b][:n] for b, n in enumerate(counts)])
        a = self.params(np.zeros((T, self.H, self.dk)), k, v)
        cu = self.d.i32(np.concatenate([[0], np.cumsum(counts)]))
        tp = self.ob.TokenPositions(cu.data_ptr(), self.d.i32([0] * len(counts)).data_ptr(), len(counts), None, None)
        self.ob.biased_attn_store(a, tp, T)

    def context(self, hist, q, plain=False, scale_out=1.0):
        """Queries q[b] behind hist[b] rows, which with their own rows make lens[b]."""
        self.fill(hist)
        counts = [len(x) for x in q]
        T = sum(counts)
        k = np.concatenate([self.k[b][h:h + n] for b, (h, n) in enumerate(zip(hist, counts))])
        v = np.concatenate([self.v[b][h:h + n] for b, (h, n) in enumerate(zip(hist, counts))])
        a = self.params(np.concatenate(q), k, v, scale_out)
        cu, hd = self.d.i32(np.concatenate([[0], np.cumsum(counts)])), self.d.i32(hist)
        tp = self.ob.TokenPositions(cu.data_ptr(), hd.data_ptr(), len(counts), None, None)
        self.ob.biased_attn_store(a, tp, T)
        self.ob.biased_attn_context(a, tp, T, max(counts), plain)
        assert self.ob.lib().onellm_gemm_timeout_flag() == 0
        return self.result()

    def decode(self, q, bound=None, scale_out=1.0):
        """The last row of every sequence is new."""
        pos = [n - 1 for n in self.lens]
        self.fill(pos)
        a = self.params(np.concatenate(q), np.stack([self.k[b][p] for b, p in enumerate(pos)]), np.stack([self.v[b][p] for b, p in enumerate(pos)]),
                        scale_out)
        step = max(self.lens)
        tp = self.ob.TokenPositions(None, None, len(pos), self.d.i32([step]).data_ptr(), self.d.i32([n - step for n in self.lens]).data_ptr())
        if self.kind == "bf16":
            ws = self.d.torch.empty(self.ob.biased_attn_decode_workspace(len(pos), self.H, self.dv), device="cuda", dtype=self.d.torch.uint8)
            self.ob.biased_attn_decode(a, tp, bound or self.S, ws)
            for b, p in enumerate(pos):  # the new rows are in the cache
                assert np.array_equal(host(self.kc[b, :, p]), self.k[b][p]) and np.array_equal(host(self.vc[b, :, p]), self.v[b][p])
        else:
            self.ob.biased_attn_store(a, tp, len(pos))
            self.ob.biased_attn_context(a, tp, len(pos), 1)
        return self.result()


@pytest.mark.parametrize("kind,plain", [("f32", False), ("bf16", True), ("bf16", False)])
@pytest.mark.parametrize("H,G,dk,dv", SIZES)
def test_attention_context(cuda, ob, kind, plain, H, G, dk, dv):
    # a whole prompt over three query tiles; a portion that starts inside a tile; two tokens behind a border
    hist, counts = [0, 37, 126], [270, 61, 2]
    t = Attn(cuda, ob, kind, H, G, dk, dv, [h + c for h, c in zip(hist, counts)], 288, seed=H + dk)
    q = t.queries(counts)
    got = t.context(hist, q, plain, scale_out=0.7)
    at = 0
    for b, (h, n) in enumerate(zip(hist, counts)):
        pick = np.unique(np.r_[0, 1, n // 2, n - 2, n - 1, np.arange(0, n, 29)])
        ref = 0.7 * t.reference(b, q[b][pick], h + pick)
        assert rel_err(got[at + pick], ref) < TOL[kind], b
        at += n


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("H,G,dk,dv", SIZES)
def test_attention_decode(cuda, ob, kind, H, G, dk, dv):
    lens = [1, 2, 16, 17, 64, 65, 130, 577]
    t = Attn(cuda, ob, kind, H, G, dk, dv, lens, 640, seed=dv)
    q = t.queries([1] * len(lens))
    got = t.decode(q, scale_out=1.5)
    for b, n in enumerate(lens):
        assert rel_err(got[b], 1.5 * t.reference(b, q[b], [n - 1])[0]) < TOL[kind], n


@pytest.mark.parametrize("B", [1, 40])
def test_attention_decode_in_one_range_and_in_many(cuda, ob, B):
    # one sequence is split over many blocks, forty fill the GPU without a split
    lens = [1500 - 31 * b for b in range(B)]
    t = Attn(cuda, ob, "bf16", 8, 8, 64, 128, lens, 1536, seed=B)
    q = t.queries([1] * B)
    got = t.decode(q)
    for b in range(0, B, 13):
        assert rel_err(got[b], t.reference(b, q[b], [lens[b] - 1])[0]) < TOL["bf16"]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 127, 128, 255, 299])
def test_one_key_that_stands_out(cuda, ob, kind, far):
    # its score is far above the others' in spite of the largest penalty: prompt and decode must both return its value
    H, G, dk, dv, n = 4, 2, 48, 64, 300
    for phase in ("context", "decode"):
        t = Attn(cuda, ob, kind, H, G, dk, dv, [n], 320, seed=far)
        q = t.queries([n if phase == "context" else 1])
        u = np.zeros(dk)
        u[5] = 12.0
        q[0][-1, :] = u
        t.k[0][:, :, 5] = 0.0
        t.k[0][far] = 4.0 * u
        got = (t.context([0], q) if phase == "context" else t.decode(q))[-1]
        ref = t.reference(0, q[0][-1:], [n - 1])[0]
        assert np.abs(ref - t.v[0][far][[0, 0, 1, 1]]).max() < 1e-3  # the case shows what it is meant to show
        assert rel_err(got, ref) < TOL[kind]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_query_temperature_at_its_edges(cuda, ob, kind):
    # the factor steps up exactly where p + 1 is a multiple of `every`; a strong coefficient makes one position off visible
    every, n = 20, 130
    t = Attn(cuda, ob, kind, 2, 2, 32, 32, [n], 144, seed=5, r1=0.0, coef=3.0, every=every)
    q = t.queries([n])
    got = t.context([0], q)
    pos = np.arange(n)
    ref = t.reference(0, q[0], pos)
    off = t.reference(0, q[0][[19, 39]], [19, 39])
    shifted = fr.biased_attention(q[0][[19, 39]], t.k[0], t.v[0], [19, 39], t.scale / fr.query_temperature(19, 3.0, every), t.r1, t.r2, 3.0, every)
    assert rel_err(shifted[0], off[0]) > 0.05
    assert rel_err(got, ref) < TOL[kind]


# ---- recurrence --------------------------------------------------------------------------------------------
def run_recurrence(ob, d, H, dk, dv, q, z, v, zb, lower, w, state, tp, B, eps=1e-5, width=None, scale_out=1.0):
    T = len(q)
    row = d.up(np.concatenate([q.reshape(T, -1), z.reshape(T, -1), v.reshape(T, -1)], 1))
    es, p = row.element_size(), row.data_ptr()
    out = d.zeros(T, H * dv + 32)
    work = d.zeros(ob.gated_recurrence_workspace(T, H, dk, dv) // 4, f32=True) + float("nan")
    g = ob.GatedRecurrence(d.dtype, H, dk, dv, p, p + H * dk * es, p + 2 * H * dk * es, row.shape[1], d.f32(zb).data_ptr(),
                           d.f32(lower).data_ptr(), d.f32(w).data_ptr(), eps, width or dv, state.data_ptr(), out.data_ptr() + 16 * es,
                           H * dv + 32, scale_out, work.data_ptr())
    ob.gated_recurrence(g, tp, T)
    o = host(out)
    assert np.all(o[:, :16] == 0) and np.all(o[:, -16:] == 0)
    return o[:, 16:-16].reshape(T, H, dv)


def ref_recurrence(q, z, v, zb, lower, w, state, eps=1e-5):
    f = fr.forget_gate(z + zb.reshape(z.shape[1:]), lower.reshape(z.shape[1:]))
    o = fr.gated_recurrence(q * fr.sigmoid(q), f, v, state)
    return fr.plain_rms_norm(o, w, eps)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("H,dk,dv", [(2, 48, 64), (3, 16, 32), (1, 128, 128), (2, 80, 96), (2, 256, 256), (4, 32, 160)])
def test_recurrence(cuda, ob, kind, H, dk, dv):
    # unequal sequences, one of them new; then a second portion behind them, down to a single token, then decode steps
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(dk + dv)
    zb = rng.uniform(-2, 9, H * dk)
    lower = rng.uniform(0, 0.95, H * dk) * (rng.uniform(size=H * dk) > 0.3)
    zb, lower = fr.round_bf16(zb), fr.round_bf16(lower)
    w = fr.round_bf16(1 + 0.3 * rng.standard_normal(dv))
    B = 3
    state = d.zeros(B, H, dk, dv, f32=True) + 1e3  # what a freed sequence left behind: a new one must not see it
    ref_state = [np.zeros((H, dk, dv)) for _ in range(B)]
    hist = [0, 0, 0]
    for counts in ([100, 1, 33], [2, 31, 64], [32, 3, 1]):
        q, z, v = (rounded(rng.standard_normal((sum(counts), H, n)) * s, kind) for n, s in ((dk, 1.0), (dk, 2.0), (dv, 1.0)))
        cu = d.i32(np.concatenate([[0], np.cumsum(counts)]))
        tp = ob.TokenPositions(cu.data_ptr(), d.i32(hist).data_ptr(), B, None, None)
        got = run_recurrence(ob, d, H, dk, dv, q, z, v, zb, lower, w, state, tp, B, scale_out=0.6)
        at = 0
        for b, n in enumerate(counts):
            s = slice(at, at + n)
            ref = 0.6 * ref_recurrence(q[s], z[s], v[s], zb, lower, w, ref_state[b])
            assert rel_err(got[s], ref) < TOL[kind], (counts, b)
            at += n
            hist[b] += n
    for i in range(4):
        q, z, v = (rounded(rng.standard_normal((B, H, n)), kind) for n in (dk, dk, dv))
        tp = ob.TokenPositions(None, None, B, d.i32([50]).data_ptr(), d.i32([0, -3, -9]).data_ptr())
        got = run_recurrence(ob, d, H, dk, dv, q, z, v, zb, lower, w, state, tp, B)
        for b in range(B):
            assert rel_err(got[b:b + 1], ref_recurrence(q[b:b + 1], z[b:b + 1], v[b:b + 1], zb, lower, w, ref_state[b])) < TOL[kind]
    # the state itself is float whatever the element type
    for b in range(B):
        assert rel_err(host(state[b]), ref_state[b]) < 2e-5


def test_recurrence_keeps_what_a_slow_gate_writes(cuda, ob):
    # a gate within 1e-5 of one: 1 - f must keep its digits, and thousands of steps must add up
    d = Dev(cuda, ob, "f32")
    H, dk, dv, T = 1, 16, 32, 3000
    zb, lower, w = np.full(dk, 11.0), np.zeros(dk), np.ones(dv)
    rng = np.random.default_rng(0)
    q = rng.uniform(0.5, 1.5, (T, H, dk)).astype(np.float32).astype(np.float64)
    v = rng.uniform(0.0, 1.0, (T, H, dv)).astype(np.float32).astype(np.float64)
    z = np.zeros((T, H, dk))
    state, rs = d.zeros(1, H, dk, dv, f32=True), np.zeros((H, dk, dv))
    tp = ob.TokenPositions(d.i32([0, T]).data_ptr(), d.i32([0]).data_ptr(), 1, None, None)
    got = run_recurrence(ob, d, H, dk, dv, q, z, v, zb, lower, w, state, tp, 1, eps=1e-12)
    assert rel_err(got, ref_recurrence(q, z, v, zb, lower, w, rs, eps=1e-12)) < 5e-5
    assert rel_err(host(state[0]), rs) < 5e-5


def test_bad_arguments_are_errors(cuda, ob):
    d = Dev(cuda, ob, "bf16")
    t = Attn(cuda, ob, "bf16", 2, 1, 32, 32, [4], 16)
    a = t.params(np.zeros((4, 2, 32)), t.k[0], t.v[0])
    tp = ob.TokenPositions(d.i32([0, 4]).data_ptr(), d.i32([0]).data_ptr(), 1, None, None)
    a.dk = 40
    with pytest.raises(ob.OnellmError) as e:
        ob.biased_attn_context(a, tp, 4, 4)
    assert e.value.status == -2
    with pytest.raises(ob.OnellmError):
        ob.project(ob.BF16, t.row, t.row, None, t.out, 4, 12, 16)
    g = ob.GatedRecurrence(ob.BF16, 1, 16, 48, 16, 16, 16, 16, 16, 16, 16, 1e-5, 48, 16, 16, 48, 1.0, 16)
    with pytest.raises(ob.OnellmError):
        ob.gated_recurrence(g, tp, 1)
