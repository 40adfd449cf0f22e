"""Every mechanism of the Fuposun design alone, against the plain statement in oracle/fuposun_ref.py, in float32 and
bfloat16.  Scores are made to stand out where random ones would hide a misplaced key."""
import numpy as np
import pytest

from oracle import fuposun_ref as ur
from oracle.finuvik_ref import plain_rms_norm, round_bf16, sigmoid
from tests.conftest import rel_err
from tests.device import Dev, host, rounded

pytestmark = pytest.mark.gpu
TOL = {"f32": 2e-5, "bf16": 1.2e-2}


def pad(n, m=16):
    return (n + m - 1) // m * m


def padded(a, width):
    """Columns behind the last one, zero."""
    return np.concatenate([a, np.zeros(a.shape[:-1] + (width - a.shape[-1],))], -1)


# ---- norms, embedding, soft cap ----------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width,ld", [(88, 96), (1024, 1024), (9000, 9008)])
def test_norm_that_takes_a_sum_of_rows_first(cuda, ob, kind, width, ld):
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(0)
    x = padded(rng.standard_normal((5, width)) * np.array([1e-3, 1, 30, 1, 0])[:, None], ld).astype(np.float32)
    w = padded(rng.standard_normal(width), ld).astype(np.float32)
    add = padded(rounded(rng.standard_normal((9, width)), kind), ld)
    rows = rng.integers(0, 9, (5, 3))
    for n_add, scale in ((0, 1.0), (1, 0.4), (3, -0.7)):
        xd, out = d.f32(x), d.zeros(5, ld)
        ref = x + scale * sum((add[rows[:, k]] for k in range(n_add)), np.zeros((5, ld)))
        kw = dict(add=d.up(add), add_rows=d.i32(rows[:, :n_add].ravel() if n_add else [0]), add_n=n_add, add_scale=scale) if n_add else {}
        ob.norm_rows(d.dtype, xd, None, 5, d.f32(w), None, out, None, 1e-5, width, ld, **kw)
        assert rel_err(host(xd), ref) < 1e-6
        assert rel_err(host(out)[:, :width], plain_rms_norm(ref[:, :width], w[:width], 1e-5)) < TOL[kind]
        assert np.all(host(out)[:, width:] == 0)
    xd = d.f32(x)  # the sum alone
    ob.norm_rows(d.dtype, xd, None, 5, None, None, None, None, 1e-5, width, ld, add=d.up(add), add_rows=d.i32(rows.ravel()), add_n=3, add_scale=2.0)
    assert rel_err(host(xd), x + 2.0 * add[rows].sum(1)) < 1e-6


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_embedding_with_a_norm(cuda, ob, kind):
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(1)
    width, ld, vocab = 41, 48, 30
    tab, w = rounded(rng.standard_normal((vocab, width)), kind), rounded(rng.standard_normal(width), kind)
    bad, out = d.i32([0, 0]), d.zeros(5, ld, f32=True) + 7
    ids = [3, 29, 0, 7, 7]
    ob.embedding_norm(d.dtype, d.i32(ids), out, d.up(padded(tab, ld)), d.f32(padded(w, ld)), 1e-3, 5, width, ld, vocab, bad)
    assert rel_err(host(out)[:, :width], plain_rms_norm(tab[ids], w, 1e-3)) < 1e-6 and np.all(host(out)[:, width:] == 0)
    assert bad.cpu().tolist() == [0, 0]
    ob.embedding_norm(d.dtype, d.i32([5, vocab, -1]), out, d.up(padded(tab, ld)), d.f32(padded(w, ld)), 1e-3, 3, width, ld, vocab, bad)
    assert bad.cpu().tolist() == [1, 0] and np.all(host(out)[1:3] == 0)


def test_softcap(cuda, ob):
    d = Dev(cuda, ob, "f32")
    x = np.random.default_rng(2).standard_normal((3, 1104)) * 40
    out = d.zeros(3, 1099, f32=True)
    ob.softcap(d.f32(x), 1104, out, 3, 1099, 7.5)
    assert rel_err(host(out), 7.5 * np.tanh(x[:, :1099].astype(np.float32) / 7.5)) < 1e-6


# ---- projections -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("M", [1, 9, 33, 64, 65, 200])
def test_clamped_gate_and_scaled_residual(cuda, ob, kind, M):
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(M)
    K, N = 80, 152
    x, w1, w2 = (rounded(rng.standard_normal(s), kind) for s in ((M, K), (K, N), (K, N)))
    y = d.zeros(M, N)
    for limit in (2.5, 30.0):
        ob.project(d.dtype, d.up(x), d.up(w1), d.up(w2), y, M, N, K, act=ob.GATE_CLAMPED, limit=limit)
        assert rel_err(host(y), ur.clamped_glu(x @ w1, x @ w2, limit)) < TOL[kind]
    r = rng.standard_normal((M, N)).astype(np.float32) * 50
    rd = d.f32(r)
    ob.project(d.dtype, d.up(x), d.up(w1), None, rd, M, N, K, f32=True, resid=rd, scale=0.3)
    assert rel_err(host(rd), 0.3 * (x @ w1) + r) < 2e-5


def test_the_clamped_gate_is_clamped_on_the_sides_it_should_be():
    # from above only, both ways, and the one added to the up value after its clamp
    assert np.isclose(ur.clamped_glu(np.array(9.0), np.array(0.0), 2.0), 2.0 / (1 + np.exp(-3.404)))
    assert np.isclose(ur.clamped_glu(np.array(-9.0), np.array(0.0), 2.0), -9.0 / (1 + np.exp(1.702 * 9)))
    assert np.isclose(ur.clamped_glu(np.array(1.0), np.array(9.0), 2.0), 3.0 / (1 + np.exp(-1.702)))
    assert np.isclose(ur.clamped_glu(np.array(1.0), np.array(-9.0), 2.0), -1.0 / (1 + np.exp(-1.702)))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("M", [1, 7, 17, 64, 100])
@pytest.mark.parametrize("H,K,N", [(3, 48, 80), (5, 16, 144), (2, 128, 512)])
def test_projection_per_head(cuda, ob, kind, M, H, K, N):
    # heads are column ranges of x and y; the weights of one layout are stacked, of the other column ranges of one matrix
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(M + H)
    x, w = rounded(rng.standard_normal((M, H, K)), kind), rounded(rng.standard_normal((H, K, N)), kind)
    ref = np.einsum("mhk,hkn->mhn", x, w)
    y = d.zeros(M, H * N + 16)
    g = ob.RowGroups(n=H, w_stride=K * N, x_stride=K, y_stride=N)
    ob.project(d.dtype, d.up(x), d.up(w), None, y, M, N, K, ldx=H * K, ldy=H * N + 16, ldw=N, groups=g)
    assert rel_err(host(y)[:, :H * N].reshape(M, H, N), ref) < TOL[kind] and np.all(host(y)[:, H * N:] == 0)
    y = d.zeros(M, H * N)
    g = ob.RowGroups(n=H, w_stride=N, x_stride=K, y_stride=N)
    ob.project(d.dtype, d.up(x), d.up(w.transpose(1, 0, 2).reshape(K, H * N)), None, y, M, N, K, ldx=H * K, ldy=H * N, ldw=H * N, groups=g)
    assert rel_err(host(y).reshape(M, H, N), ref) < TOL[kind]


# ---- experts -----------------------------------------------------------------------------------------------
class Routing:
    def __init__(self, ob, d, T, E, top, logits, ld, x=None):
        self.T, self.E, self.top = T, E, top
        n = T * top
        tiles = ob.route_max_tiles(T, E, top)
        self.a = {k: d.i32(np.full(s, -7)) for k, s in (("slot", n), ("slot_token", n), ("off", E + 1), ("used", min(E, n)), ("n_used", 1),
                                                         ("tile_group", tiles), ("tile_row", tiles), ("n_tiles", 1), ("choice", n))}
        self.a.update(slot_weight=d.zeros(n, f32=True), choice_weight=d.zeros(n, f32=True), count=d.i32(np.zeros(E)), logits=d.f32(logits))
        self.r = ob.Route(T, E, top, ld=ld, dtype=d.dtype, **{k: v.data_ptr() for k, v in self.a.items()})
        self.xs = None
        if x is not None:
            self.xs = d.zeros(n, x.shape[1])
            self.r.x, self.r.xs, self.r.ld_x = x.data_ptr(), self.xs.data_ptr(), x.shape[1]
        ob.route(self.r)
        ob.route(self.r)  # the scratch is left as it was found
        self.max_tiles = tiles
        for k, v in self.a.items():
            setattr(self, k, v.cpu().numpy())


@pytest.mark.parametrize("E,top", [(1, 1), (3, 3), (11, 1), (40, 4), (130, 8), (1024, 2)])
@pytest.mark.parametrize("T", [1, 5, 64, 65, 700])
def test_routing(cuda, ob, T, E, top):
    d = Dev(cuda, ob, "f32")
    rng = np.random.default_rng(T + E)
    ld = pad(E, 8) + 8
    z = np.full((T, ld), 1e9, np.float32)  # columns behind the experts take no part
    z[:, :E] = rng.standard_normal((T, E)) * 3 + 2 * rng.standard_normal(E)
    z[0, :E] = 0.5  # ties go to the lower number
    if T > 3:
        z[3, :E] = np.where(np.arange(E) % 2, 1.0, -1.0)
    x = d.f32(rng.standard_normal((T, 24))) if T > 64 else None
    r = Routing(ob, d, T, E, top, z, ld, x)
    s = sigmoid(z[:, :E].astype(np.float64))
    chosen = np.argsort(-z[:, :E], 1, kind="stable")[:, :top]
    slot = r.slot.reshape(T, top)
    assert sorted(r.slot.tolist()) == list(range(T * top))
    expert_of = np.searchsorted(r.off, slot, side="right") - 1
    assert np.array_equal(expert_of, chosen)
    assert np.array_equal(r.slot_token[slot], np.repeat(np.arange(T)[:, None], top, 1))
    assert rel_err(r.slot_weight[slot], np.take_along_axis(s, chosen, 1)) < 1e-6
    counts = np.bincount(chosen.ravel(), minlength=E)
    assert np.array_equal(np.diff(r.off), counts) and r.off[0] == 0
    assert np.array_equal(r.used[:r.n_used[0]], np.flatnonzero(counts))
    tiles = [(e, r.off[e] + i) for e in range(E) for i in range(0, counts[e], 128)]
    assert r.n_tiles[0] == len(tiles) <= r.max_tiles
    assert [(a, b) for a, b in zip(r.tile_group[:len(tiles)], r.tile_row)] == tiles
    assert np.all(r.count == 0)
    if x is not None:
        assert np.array_equal(host(r.xs), host(x)[r.slot_token])


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("E,top,W,ff", [(6, 1, 96, 48), (9, 3, 80, 144), (33, 2, 272, 176)])
@pytest.mark.parametrize("T", [1, 8, 33, 64, 65, 300])
def test_mixture_of_experts(cuda, ob, kind, T, E, top, W, ff):
    """Routing, gate and up with the weight in front of the gate function, down, and the sum over a token's experts."""
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(T + E)
    lim = 1.2
    h = rounded(rng.standard_normal((T, W)), kind)
    router = rounded(rng.standard_normal((E, W)) / np.sqrt(W), kind)
    router[E // 2] *= 4  # one expert that many tokens choose, some that none does
    ws = [[rounded(rng.standard_normal(s) / np.sqrt(s[1]) * a, kind) for s, a in (((ff, W), 2.0), ((ff, W), 2.0), ((W, ff), 1.0))] for _ in range(E)]
    hd = d.up(h)
    r = Routing(ob, d, T, E, top, h @ router.T, E, hd if T > 64 else None)
    tiled = T > 64 and kind == "bf16"
    gate, up, down = (d.up(np.stack([w[i].T for w in ws])) for i in range(3))
    act, ys = d.zeros(T * top, ff), d.zeros(T * top, W)
    a = {k: v.data_ptr() for k, v in r.a.items()}
    g = ob.RowGroups(n=E if tiled else min(E, T * top), used=None if tiled else a["used"], n_used=None if tiled else a["n_used"], off=a["off"],
                     x_rows=None if tiled else a["slot_token"], row_scale=a["slot_weight"], w_stride=W * ff, tile_group=a["tile_group"],
                     tile_row=a["tile_row"], n_tiles=a["n_tiles"], max_tiles=r.max_tiles, weights=E, rows=T * top)
    ob.project(d.dtype, r.xs if tiled else hd, gate, up, act, T, ff, W, act=ob.GATE_CLAMPED, limit=lim, groups=g)
    g.x_rows, g.row_scale = None, None
    ob.project(d.dtype, act, down, None, ys, T, W, ff, groups=g)
    x = d.zeros(T, W, f32=True)
    ob.norm_rows(d.dtype, x, None, T, None, None, None, None, 1e-5, W, W, add=ys, add_rows=r.a["slot"], add_n=top, add_scale=0.5)
    assert ob.lib().onellm_gemm_timeout_flag() == 0
    ref = 0.5 * ur.mixture(h, router, top, ws, lim)
    assert rel_err(host(x), ref) < TOL[kind]
    # a weight on the output instead would show
    chosen, w = ur.route(h, router, top)
    other = [0.5 * sum(w[t, k] * ur.expert(h[t:t + 1], *ws[chosen[t, k]], lim)[0] for k in range(top)) for t in range(T)]
    assert rel_err(other, ref) > 0.03


# ---- attention over latents --------------------------------------------------------------------------------
class Latents:
    """Rings of B sequences behind a window, filled through the store kernels, and the parameters of a launch.  Position j of
    sequence b has the raw latent raw[b][j]; what is cached is its norm."""

    def __init__(self, cuda, ob, kind, H, rank, window, lens, seed=0, R=None):
        self.ob, self.kind, self.d, self.torch = ob, kind, Dev(cuda, ob, kind), cuda
        self.H, self.rank, self.rp, self.window, self.lens = H, rank, pad(rank, 64), window, lens
        rng = self.rng = np.random.default_rng(seed)
        self.w = round_bf16(1 + 0.2 * rng.standard_normal(rank))
        self.qw = round_bf16(1 + 0.2 * rng.standard_normal(24))
        self.raw = [rounded(rng.standard_normal((n, rank)), kind) for n in lens]
        self.R = R or window
        # unused rows hold what a freed sequence may leave behind
        self.ring = self.d.zeros(len(lens), self.R, self.rp) + float("nan")
        self.scale = 1.5 / np.sqrt(rank)

    def latents(self, b):
        return rounded(plain_rms_norm(self.raw[b], self.w, 1e-5), self.kind)

    def store(self, hist, counts, joined=False, decode=False):
        """Tokens hist[b] .. hist[b] + counts[b] of every sequence through the store kernel; also normed queries of width 24."""
        d = self.d
        T = sum(counts)
        kv = np.concatenate([self.raw[b][h:h + n] for b, (h, n) in enumerate(zip(hist, counts))])
        qin = rounded(self.rng.standard_normal((T, 24)), self.kind)
        self.row = d.up(np.concatenate([padded(qin, 32), padded(kv, self.rp)], 1))
        es = self.row.element_size()
        self.q_out = d.zeros(T, 32)
        kept = [min(h, self.window - 1) for h in hist]
        self.fresh = d.zeros(T + sum(kept), self.rp) + float("nan")
        a = self.a = self.ob.LatentAttn(d.dtype, self.H, self.rank, self.window, self.R, self.ring.data_ptr(), self.fresh.data_ptr(), joined,
                                        self.row.data_ptr(), self.row.data_ptr() + 32 * es, self.row.shape[1], d.f32(padded(self.qw, 32)).data_ptr(),
                                        d.f32(padded(self.w, self.rp)).data_ptr(), 24, 32, self.q_out.data_ptr(), 1e-5)
        if decode:
            step = max(h + 1 for h in hist)
            self.tp = self.ob.TokenPositions(None, None, len(hist), d.i32([step]).data_ptr(), d.i32([h + 1 - step for h in hist]).data_ptr())
        else:
            self.tp = self.ob.TokenPositions(d.i32(np.concatenate([[0], np.cumsum(counts)])).data_ptr(), d.i32(hist).data_ptr(), len(hist), None, None)
        self.ob.latent_store(a, self.tp, T, max(hist))
        assert rel_err(host(self.q_out)[:, :24], plain_rms_norm(qin, self.qw, 1e-5)) < TOL[self.kind]
        assert np.all(host(self.q_out)[:, 24:] == 0)
        self.counts = counts

    def keep(self):
        self.ob.latent_keep(self.a, self.tp, max(self.counts))

    def attend(self, q, gate=None, plain=False, out_scale=1.0):
        d, T = self.d, len(q)
        out = d.zeros(T, self.H, self.rp) + float("nan")
        a = self.a
        a.q, a.scale, a.out, a.out_scale = d.up(padded(q, self.rp)).data_ptr(), self.scale, out.data_ptr(), out_scale
        if gate is not None:
            a.gate, a.gate_ld = d.up(gate).data_ptr(), gate.shape[1]
        ws = self.torch.empty(self.ob.latent_attn_workspace(T, self.H, self.rank), device="cuda", dtype=self.torch.uint8)
        self.ob.latent_attn(a, self.tp, T, max(self.lens), ws, plain)
        o = host(out)
        assert np.all(o[:, :, self.rank:] == 0)
        return o[:, :, :self.rank]

    def reference(self, b, q, pos):
        """Keys and values are the latents themselves: identity matrices in front of the plain statement."""
        eye = np.tile(np.eye(self.rank), (self.H, 1))
        c = self.latents(b)[:max(pos) + 1]
        return ur.latent_attention(q, c, eye, eye, pos, np.arange(len(c)), self.scale, self.window)


LATENT_SIZES = [(1, 16, 5), (8, 96, 33), (20, 72, 1), (16, 144, 64), (3, 272, 100), (17, 512, 40), (2, 1024, 31), (4, 128, 700), (70, 64, 300)]  # H, rank, window


@pytest.mark.parametrize("kind,plain", [("f32", True), ("bf16", True), ("bf16", False)])
@pytest.mark.parametrize("H,rank,window", LATENT_SIZES)
def test_latent_attention(cuda, ob, kind, plain, H, rank, window):
    # portions behind unequal histories, cut anywhere, rings that wrap several times, then decode steps
    t = Latents(cuda, ob, kind, H, rank, window, [194, 16, 133, 800], seed=H + rank)
    hist = [0, 0, 0, 0]
    for counts in ([10, 1, 40, 13], [2, 2, 3, 50]):
        q = rounded(t.rng.standard_normal((sum(counts), H, rank)), kind)
        gate = rounded(t.rng.standard_normal((sum(counts), H + 3)), kind)
        t.store(hist, counts)
        got = t.attend(q, gate, plain, 0.7)
        t.keep()
        at = 0
        for b, n in enumerate(counts):
            ref = 0.7 * sigmoid(gate[at:at + n, :H])[:, :, None] * t.reference(b, q[at:at + n], hist[b] + np.arange(n))
            assert rel_err(got[at:at + n], ref) < TOL[kind], (counts, b)
            at += n
            hist[b] += n
    # the rest of the sequences without looking, in one portion longer than the window and in pieces of it
    t.store(hist, [100, 1, 80, 600])
    t.keep()
    hist = [h + n for h, n in zip(hist, [100, 1, 80, 600])]
    t.store(hist, [77, 7, 5, 130])
    t.keep()
    hist = [h + n for h, n in zip(hist, [77, 7, 5, 130])]
    for _ in range(5):
        q = rounded(t.rng.standard_normal((4, H, rank)), kind)
        t.store(hist, [1] * 4, decode=True)
        got = t.attend(q, None, plain)
        for b in range(4):
            assert rel_err(got[b:b + 1], t.reference(b, q[b:b + 1], [hist[b]])) < TOL[kind], b
        hist = [h + 1 for h in hist]


@pytest.mark.parametrize("kind,plain", [("f32", True), ("bf16", True), ("bf16", False)])
@pytest.mark.parametrize("phase", ["portion", "decode"])
@pytest.mark.parametrize("window", [1, 2, 32, 33, 50, 129])
def test_the_edge_of_the_window(cuda, ob, kind, plain, phase, window):
    """A key far above all others at the last distance the window has, and at the first it has not."""
    n, H, rank = 170, 4, 48
    for dist in (window - 1, window):
        t = Latents(cuda, ob, kind, H, rank, window, [n], seed=window)
        far = n - 1 - dist
        c = t.latents(0)
        q = rounded(np.tile(25.0 * c[far], (1, H, 1)), kind)
        q = np.concatenate([rounded(t.rng.standard_normal((2, H, rank)), kind), q]) if phase == "portion" else q
        k = len(q)
        t.store([0], [n - k])
        t.keep()
        t.store([n - k], [k], decode=phase == "decode")
        got = t.attend(q, None, plain)[-1]
        ref = t.reference(0, q[-1:], [n - 1])[0]
        assert (rel_err(ref, np.tile(c[far], (H, 1))) < 1e-3) == (dist < window)  # the case shows what it is meant to show
        assert rel_err(got, ref) < TOL[kind], dist


def test_latent_attention_in_one_range_and_in_many(cuda, ob):
    for B, window in ((1, 3000), (33, 500)):
        t = Latents(cuda, ob, "bf16", 6, 128, window, [3500 - 40 * b for b in range(B)], seed=B)
        hist = [n - 1 for n in t.lens]
        t.store([0] * B, hist)
        t.keep()
        q = rounded(t.rng.standard_normal((B, 6, 128)), "bf16")
        t.store(hist, [1] * B, decode=True)
        got = t.attend(q)
        for b in range(0, B, 8):
            assert rel_err(got[b:b + 1], t.reference(b, q[b:b + 1], [hist[b]])) < TOL["bf16"]


@pytest.mark.parametrize("H,dk,dv,window", [(2, 16, 32, 1), (3, 48, 80, 7), (2, 64, 128, 64), (2, 128, 64, 65), (1, 256, 256, 200), (4, 80, 112, 128),
                                            (2, 64, 64, 1000)])
def test_window_attention_of_a_context_pass(cuda, ob, H, dk, dv, window):
    """Keys and values formed from the joined latents; queries over several tiles, portions behind a history, both edges."""
    rank, rp = 48, 64
    lens = [290, 61, 130, 2]
    hist = [0, 37, 126, 0]
    counts = [n - h for n, h in zip(lens, hist)]
    t = Latents(cuda, ob, "bf16", H, rank, window, lens, seed=dk)
    d = t.d
    t.store([0] * 4, [max(h, 0) for h in hist])
    t.keep()
    t.store(hist, counts, joined=True)
    uk, uv = (rounded(t.rng.standard_normal((H * n, rank)) / np.sqrt(rank), "bf16") for n in (dk, dv))
    ld, rows = H * (dk + dv), t.fresh.shape[0]
    kv = d.zeros(rows, ld)
    ob.project(ob.BF16, t.fresh, d.up(padded(np.concatenate([uk, uv]), rp).T), None, kv, rows, ld, rp)
    T = sum(counts)
    q = rounded(t.rng.standard_normal((T, H, dk)) * 2, "bf16")
    # one key that stands out at the last visible distance of the first sequence's last query, another just outside
    c, last = t.latents(0), counts[0] - 1
    if last - window >= 0:
        k = rounded(c @ uk.T, "bf16").reshape(-1, H, dk)
        q[last] = 6 * (k[last - window + 1] + 2 * k[last - window])
        q = rounded(q, "bf16")
    gate = rounded(t.rng.standard_normal((T, 8)), "bf16")
    out = d.zeros(T, H * dv + 16)
    a = ob.WindowAttn(H, dk, dv, window, d.up(q).data_ptr(), H * dk, kv.data_ptr(), ld, rows, 0.2, d.up(gate).data_ptr(), 8, out.data_ptr(),
                      H * dv + 16, 0.6)
    ob.window_attn(a, t.tp, max(counts))
    assert ob.lib().onellm_gemm_timeout_flag() == 0
    got = host(out)
    assert np.all(got[:, H * dv:] == 0)
    got = got[:, :H * dv].reshape(T, H, dv)
    at = 0
    for b, (h, n) in enumerate(zip(hist, counts)):
        pick = np.unique(np.r_[0, 1, n // 2, max(n - 2, 0), n - 1, np.arange(0, n, 23)])
        pick = pick[pick < n]
        ref = ur.latent_attention(q[at + pick], t.latents(b), uk, uv, h + pick, np.arange(lens[b]), 0.2, window)
        ref *= 0.6 * sigmoid(gate[at + pick, :H])[:, :, None]
        assert rel_err(got[at + pick], ref) < 1.5 * TOL["bf16"], b
        at += n
    t.keep()  # the ring holds the last positions of every sequence
    ring = host(t.ring)
    for b, n in enumerate(lens):
        for j in range(max(0, n - window), n):
            assert rel_err(ring[b, j % window, :rank], t.latents(b)[j]) < TOL["bf16"]


# ---- gated linear attention --------------------------------------------------------------------------------
def run_gla(ob, d, H, dk, dv, x, A, zb, w, state, tp, tau, q_scale, eps=1e-5, width=None, scale_out=1.0, gated=True):
    q, k, v, r, g = x
    T, rank = len(q), r.shape[1]
    parts = [q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), g.reshape(T, -1), padded(r, pad(rank, 8))]
    row = d.up(np.concatenate(parts, 1))
    es, at, ptr = row.element_size(), 0, []
    for p in parts:
        ptr.append(row.data_ptr() + at * es)
        at += p.shape[1]
    out = d.zeros(T, H * dv + 32)
    work = d.zeros(ob.gated_recurrence_workspace(T, H, dk, dv, ob.GR_KEYED) // 4, f32=True) + float("nan")
    a = ob.GatedRecurrence(d.dtype, H, dk, dv, q=ptr[0], v=ptr[2], ld=at, zb=d.f32(zb).data_ptr(), w=d.f32(w).data_ptr(), eps=eps, norm_width=width or dv,
                           state=state.data_ptr(), out=out.data_ptr() + 16 * es, out_ld=H * dv + 32, out_scale=scale_out, work=work.data_ptr(),
                           kind=ob.GR_KEYED, k=ptr[1], r=ptr[4], rank=rank, A=d.f32(A).data_ptr(), inv_tau=1.0 / tau, q_scale=q_scale,
                           g=ptr[3] if gated else None)
    ob.gated_recurrence(a, tp, T)
    assert ob.lib().onellm_gemm_timeout_flag() == 0
    o = host(out)
    assert np.all(o[:, :16] == 0) and np.all(o[:, -16:] == 0)
    return o[:, 16:-16].reshape(T, H, dv)


def ref_gla(x, A, zb, w, state, tau, q_scale, eps=1e-5, gated=True):
    q, k, v, r, g = x
    alpha = ur.channel_decay(r @ A.T + zb, tau).reshape(q.shape)
    o = plain_rms_norm(ur.gated_linear_attention(q * q_scale, k, v, alpha, state), w, eps)
    return o * ur.silu(g) if gated else o


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("H,dk,dv,rank", [(2, 48, 64, 16), (3, 16, 32, 5), (1, 128, 128, 1), (2, 80, 96, 33), (2, 256, 512, 16), (1, 320, 32, 8),
                                          (1, 512, 320, 16), (4, 32, 160, 7), (1, 16, 1280, 4)])
def test_gated_linear_attention(cuda, ob, kind, H, dk, dv, rank):
    # unequal sequences, one of them new; then further portions down to a single token, then decode steps
    d = Dev(cuda, ob, kind)
    rng = np.random.default_rng(dk + dv)
    A, zb = (round_bf16(x) for x in (rng.standard_normal((H * dk, rank)) / np.sqrt(rank), rng.uniform(-1, 6, H * dk)))
    w, tau, qs = round_bf16(1 + 0.3 * rng.standard_normal(dv)), 3.0, dk ** -0.5
    B = 3
    state = d.zeros(B, H, dk, dv, f32=True) + float("nan")  # what a freed sequence left behind: a new one must not see it
    ref_state = [np.zeros((H, dk, dv)) for _ in range(B)]
    draw = lambda T: tuple(rounded(rng.standard_normal(s), kind) for s in ((T, H, dk), (T, H, dk), (T, H, dv), (T, rank), (T, H, dv)))
    hist = [0, 0, 0]
    for counts in ([100, 1, 33], [2, 31, 64], [32, 3, 1]):
        x = draw(sum(counts))
        tp = ob.TokenPositions(d.i32(np.concatenate([[0], np.cumsum(counts)])).data_ptr(), d.i32(hist).data_ptr(), B, None, None)
        got = run_gla(ob, d, H, dk, dv, x, A, zb, w, state, tp, tau, qs, scale_out=0.6)
        at = 0
        for b, n in enumerate(counts):
            ref = 0.6 * ref_gla([y[at:at + n] for y in x], A, zb, w, ref_state[b], tau, qs)
            assert rel_err(got[at:at + n], ref) < TOL[kind], (counts, b)
            at += n
            hist[b] += n
    for i in range(4):
        x = draw(B)
        tp = ob.TokenPositions(None, None, B, d.i32([50]).data_ptr(), d.i32([0, -3, -9]).data_ptr())
        got = run_gla(ob, d, H, dk, dv, x, A, zb, w, state, tp, tau, qs, gated=i % 2 == 0)
        for b in range(B):
            assert rel_err(got[b:b + 1], ref_gla([y[b:b + 1] for y in x], A, zb, w, ref_state[b], tau, qs, gated=i % 2 == 0)) < TOL[kind]
    for b in range(B):  # the state itself is float whatever the element type
        assert rel_err(host(state[b]), ref_state[b]) < 2e-5


def test_a_decode_step_at_the_first_position_starts_from_zero(cuda, ob):
    d = Dev(cuda, ob, "f32")
    rng = np.random.default_rng(3)
    x = tuple(rng.standard_normal(s).astype(np.float32).astype(np.float64) for s in ((1, 2, 32), (1, 2, 32), (1, 2, 64), (1, 4), (1, 2, 64)))
    A, zb, w = rng.standard_normal((64, 4)).astype(np.float32), np.zeros(64), np.ones(64)
    state = d.zeros(1, 2, 32, 64, f32=True) + float("nan")
    tp = ob.TokenPositions(None, None, 1, d.i32([1]).data_ptr(), d.i32([0]).data_ptr())
    got = run_gla(ob, d, 2, 32, 64, x, A, zb, w, state, tp, 16.0, 1.0)
    assert rel_err(got, ref_gla(x, A, zb, w, np.zeros((2, 32, 64)), 16.0, 1.0)) < 2e-5


def test_gated_linear_attention_remembers_through_a_slow_decay(cuda, ob):
    # a decay within 1e-6 of one (a large tau): what the first tokens wrote must still be there after thousands
    d = Dev(cuda, ob, "f32")
    H, dk, dv, T, tau = 1, 16, 32, 3000, 500.0
    rng = np.random.default_rng(0)
    f32 = lambda a: a.astype(np.float32).astype(np.float64)
    k = f32(rng.standard_normal((T, H, dk)))
    k[5:] *= 1e-3
    x = (f32(rng.uniform(0.5, 1.5, (T, H, dk))), k, f32(rng.standard_normal((T, H, dv))), np.zeros((T, 3)), f32(rng.standard_normal((T, H, dv))))
    A, zb, w = np.zeros((dk, 3)), np.full(dk, 8.0), np.ones(dv)
    state, rs = d.zeros(1, H, dk, dv, f32=True), np.zeros((H, dk, dv))
    tp = ob.TokenPositions(d.i32([0, T]).data_ptr(), d.i32([0]).data_ptr(), 1, None, None)
    got = run_gla(ob, d, H, dk, dv, x, A, zb, w, state, tp, tau, 0.25)
    ref = ref_gla(x, A, zb, w, rs, tau, 0.25)
    assert np.abs(rs).max() > 0.5
    # a state moves by a dozen of its float steps at a time here, whose rounding adds up
    assert rel_err(host(state[0]), rs) < 3e-4 and rel_err(got, ref) < 3e-4


def test_bad_arguments_are_errors(cuda, ob):
    d = Dev(cuda, ob, "bf16")
    y = d.zeros(8, 64)
    g = ob.RowGroups(n=2, w_stride=12, x_stride=16, y_stride=16)
    with pytest.raises(ob.OnellmError):  # strides that the kernels do not take
        ob.project(ob.BF16, y, y, None, y, 4, 16, 16, ldx=64, ldy=64, groups=g)
    with pytest.raises(ob.OnellmError):  # strides without groups
        ob.project(ob.BF16, y, y, None, y, 4, 16, 16, ldx=64)
    with pytest.raises(ob.OnellmError):  # more than 64 rows per group without a tile table
        ob.project(ob.BF16, y, y, None, y, 65, 16, 16, groups=ob.RowGroups(n=1, off=y.data_ptr(), w_stride=256))
    with pytest.raises(ob.OnellmError):
        ob.route(ob.Route(4, 2000, 1, ld=2000))
    t = Latents(cuda, ob, "bf16", 2, 48, 4, [4])
    t.store([0], [4])
    t.a.rank = 1100
    with pytest.raises(ob.OnellmError) as e:
        ob.latent_attn(t.a, t.tp, 4, 4, y)
    assert e.value.status == -1 or e.value.status == -2
    with pytest.raises(ob.OnellmError):
        ob.window_attn(ob.WindowAttn(1, 40, 40, 4, 16, 40, 16, 80, 4, 1.0, None, 0, 16, 40, 1.0), t.tp, 4)
