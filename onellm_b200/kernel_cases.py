"""One hot kernel (or one fixed sequence of them) alone on a fixed case: the micro-benchmark behind the
per-kernel figures of `bench.py` and the target of every `ncu` capture summarised under `profiles/`.

    python -m onellm_b200.kernel_cases <case> [--model 7b|13b] [--batch B] [--ctx C] [--tp T] [--iters N] [--graph] [--plain]

Decode-step cases (HBM-bound, reported in GB/s of algorithmic bytes):
    qkv, o_proj, gate_up, down     the four projections as the decode step runs them (onellm_gemm_fused: RMS scale
                                   or residual add in the kernel); --plain times onellm_gemm / onellm_gemm_swiglu
    lm_head_kn, lm_head            LM head on the [hidden, vocab] copy the model keeps / on [vocab, hidden]
    attn                           decode attention over a cache of --ctx rows
    attn_c1                        the fp32 unit-test shape: batch 2, 32 heads x 128, step 255
    norm, rmsnorm                  fused add-residual RMSNorm / RMSNorm on 4096 x hidden fp16
    norm8                          the same on --batch rows
    topk, sample                   top-K (K = 50) over [batch, vocab] fp16 logits / the sampler behind it
    decode_layer                   the five kernels of one decoder layer in the decode step's order (QKV, attention, o_proj,
                                   gate/up, down); with --graph: the layer as the decode step runs it
Context-phase cases (reported in TFLOP/s, except prefill_rope):
    prefill_qkv, prefill_o, prefill_gate, prefill_down, prefill_lm     projections on --batch x --ctx token rows
    prefill_attn                   causal attention of --batch sequences x --ctx tokens
    prefill_rope                   bias + RoPE + KV-cache write (GB/s)
    prefill_layer                  one whole decoder layer on --batch x --ctx tokens as the model runs it: QKV projection (RMS scale
                                   in its epilogue), RoPE + cache write, attention, o_proj (+ residual), gate/up + SwiGLU, down (+ residual)

Cases of the mechanisms behind onellm_model_open (bfloat16; widths and heads of --model, keys and values of head_size, as
many recurrence heads as attention heads), each beside the like case above:
    fv_mix, fv_gate_up, fv_out     decode: all mixer projections at once, ReLU-gated pair, stacked output projections added to
                                   the float stream
    fv_attn, fv_rec, fv_norm       decode attention with factor and penalty tables; one recurrence step; two norms of a float
                                   stream of 4096 rows
    prefill_fv_mix, prefill_fv_gate, prefill_fv_out, prefill_fv_attn, prefill_fv_rec       the same in the context phase

    fu_in, fu_uq, fu_out           decode: mixer inputs of a gla layer, queries out of their latent, output added to the float stream
    fu_absorb, fu_attn, fu_uv      queries into latent space per head, attention over a window of --ctx latents, values out of it
    fu_rec, fu_norm                one step of the gla recurrence; norm of 4096 rows that takes the experts' rows first
    fu_route, fu_egate, fu_edown   router and choice; gate/up and down of the chosen experts
    prefill_fu_in, prefill_fu_kv, prefill_fu_attn, prefill_fu_rec, prefill_fu_route, prefill_fu_egate, prefill_fu_edown
                                   the same in the context phase (window: 1024 positions)

Every case holds a few hundred MB on the device (more than the 126 MB L2, far less than a model) and runs on
rotating buffers.  `--tp T` uses the per-rank shapes of T-way tensor parallelism; `--graph` times the launches as
one CUDA graph, i.e. back to back on the device without the host's launch cost (what a decode step sees).
"""
from __future__ import annotations

import argparse
from dataclasses import dataclass
from typing import Callable

import onellm_b200 as ob

MODELS = {
    "7b": dict(hidden=4096, head_num=32, head_size=128, inter_size=11008, vocab_size=32000),
    "13b": dict(hidden=5120, head_num=40, head_size=128, inter_size=13824, vocab_size=32000),
}

DECODE_CASES = ["qkv", "o_proj", "gate_up", "down", "lm_head_kn", "lm_head", "attn", "attn_c1", "norm", "rmsnorm", "norm8",
                "topk", "sample", "decode_layer", "fv_mix", "fv_gate_up", "fv_out", "fv_attn", "fv_rec", "fv_norm", "fu_in", "fu_uq", "fu_out",
                "fu_absorb", "fu_attn", "fu_uv", "fu_rec", "fu_norm", "fu_route", "fu_egate", "fu_edown"]
PREFILL_CASES = ["prefill_qkv", "prefill_o", "prefill_gate", "prefill_down", "prefill_lm", "prefill_attn", "prefill_rope",
                 "prefill_layer", "prefill_fv_mix", "prefill_fv_gate", "prefill_fv_out", "prefill_fv_attn", "prefill_fv_rec", "prefill_fu_in",
                 "prefill_fu_kv", "prefill_fu_attn", "prefill_fu_rec", "prefill_fu_route", "prefill_fu_egate", "prefill_fu_edown"]


@dataclass
class Case:
    fn: Callable[[int], None]   # fn(i) launches the case on rotating buffer set i
    rot: int                    # number of buffer sets
    amount: float               # algorithmic bytes (unit "B") or flops (unit "flop") per call of fn
    unit: str
    kernel: str                 # the kernel that dominates the case
    launches: int = 1           # kernel launches per call of fn
    keep: tuple = ()            # buffers kept alive


def _projection_kernel(tokens, dual):
    """Name of the kernel a [K, N] projection of `tokens` rows runs on."""
    if tokens >= ob.gemm_tc_min_tokens() and tokens <= 64:
        return f"skinny_tc_kernel<{'true' if dual else 'false'}>"
    mb = 1 if tokens <= 8 else 2 if tokens <= 16 else 4 if tokens <= 32 else 8
    return f"skinny_kn_staged_kernel<{mb},{'true' if dual else 'false'},false>"


def make_mechanism_case(name, torch, m, B, ctx, plain=False) -> Case:
    """The fv_ cases: m as in MODELS, optionally with kv_heads, value_size, rec_heads, rec_key, rec_value."""
    prefill = name.startswith("prefill_")
    what = name.rsplit("_", 1)[1] if not name.endswith("gate_up") else "gate"
    W, H, D, INTER = m["hidden"], m["head_num"], m["head_size"], m["inter_size"]
    G, DV = m.get("kv_heads", H), m.get("value_size", D)
    RH, RK, RV = m.get("rec_heads", H), m.get("rec_key", D), m.get("rec_value", D)
    n_mix = (H + G) * D + G * DV + RH * (2 * RK + RV)
    n_cat = H * DV + RH * RV + INTER
    T = B * ctx if prefill else B
    bf = dict(device="cuda", dtype=torch.bfloat16)
    f32 = dict(device="cuda", dtype=torch.float32)
    rnd = lambda *s: 0.02 * torch.randn(*s, **bf)
    n_rot = lambda nbytes, target=400e6: 2 if prefill else max(2, int(target // nbytes) + 1)
    BF = ob.BF16
    if what in ("mix", "gate", "out"):
        K, N = {"mix": (W, n_mix), "gate": (W, INTER), "out": (n_cat, W)}[what]
        dual = what == "gate"
        rot = n_rot(K * N * 2 * (2 if dual else 1))
        x, w = torch.randn(T, K, **bf), [rnd(K, N) for _ in range(rot)]
        wu = [rnd(K, N) for _ in range(rot)] if dual else [None] * rot
        if what == "out":
            y = torch.randn(T, N, **f32)
            fn = lambda i: ob.project(BF, x, w[i], None, y, T, N, K, f32=True, resid=y)
        elif dual:
            y = torch.zeros(T, n_cat, **bf)
            fn = lambda i: ob.project(BF, x, w[i], wu[i], y.data_ptr() + (n_cat - INTER) * 2, T, N, K, ldy=n_cat, act=ob.GATE_RELU)
        else:
            y = torch.zeros(T, N, **bf)
            fn = lambda i: ob.project(BF, x, w[i], None, y, T, N, K)
        if prefill:
            return Case(fn, rot, 2.0 * T * N * K * (2 if dual else 1), "flop", "gemm_tc_kernel (bf16)", keep=(x, w, wu, y))
        nbytes = K * N * 2 * (2 if dual else 1) + T * K * 2 + T * N * (8 if what == "out" else 2)
        return Case(fn, rot, nbytes, "B", _projection_kernel(T, dual) + " (bf16)", keep=(x, w, wu, y))
    if what == "norm":
        rows = 4096
        xs = [torch.randn(rows, W, **f32) for _ in range(4)]
        w1, w2, o1, o2 = torch.zeros(W, **f32), torch.zeros(W, **f32), torch.empty(rows, W, **bf), torch.empty(rows, W, **bf)
        fn = lambda i: ob.norm_rows(BF, xs[i], None, rows, w1, w2, o1, o2, 1e-6, W, W, w_base=1.0)
        return Case(fn, 4, rows * W * 8, "B", "norm_rows_kernel", keep=(xs, w1, w2, o1, o2))
    mix, cat = torch.randn(T, n_mix, **bf), torch.zeros(T, n_cat, **bf)
    cu = torch.arange(0, B + 1, device="cuda", dtype=torch.int32) * ctx
    hist, off = torch.zeros(B, device="cuda", dtype=torch.int32), torch.zeros(B, device="cuda", dtype=torch.int32)
    step = torch.full((1,), ctx + 1, device="cuda", dtype=torch.int32)
    tp = ob.TokenPositions(cu.data_ptr(), hist.data_ptr(), B, None, None) if prefill else \
        ob.TokenPositions(None, None, B, step.data_ptr(), off.data_ptr())
    p = mix.data_ptr()
    if what == "attn":
        S = max(2048, ctx + 8)
        rot = n_rot(B * G * S * (D + DV) * 2, 300e6)
        kc, vc = [torch.randn(B, G, S, D, **bf) for _ in range(rot)], [torch.randn(B, G, S, DV, **bf) for _ in range(rot)]
        qf, pen = torch.empty(S, **f32), torch.empty(H, S, **f32)
        ob.query_factor(qf, S, D ** -0.5, 0.1, 1024)
        ob.distance_penalty(pen, torch.ones(H, **f32), torch.full((H,), 0.1, **f32), H, S)
        a = [ob.BiasedAttn(BF, H, G, D, DV, p, p + H * D * 2, p + (H + G) * D * 2, n_mix, kc[i].data_ptr(), vc[i].data_ptr(), S,
                           qf.data_ptr(), pen.data_ptr(), cat.data_ptr(), n_cat, 1.0) for i in range(rot)]
        ws = torch.empty(ob.biased_attn_decode_workspace(B, H, DV), device="cuda", dtype=torch.uint8)
        keep = (mix, cat, cu, hist, off, step, kc, vc, qf, pen, ws)
        if prefill:
            fn = lambda i: ob.biased_attn_context(a[i], tp, T, ctx, plain)
            return Case(fn, rot, float(B * H * 2 * (D + DV) * ctx * (ctx + 1) / 2), "flop", "biased_attn_tc_kernel", keep=keep)
        fn = lambda i: ob.biased_attn_decode(a[i], tp, ctx + 1, ws)
        nbytes = ctx * B * G * (D + DV) * 2 + B * (H * D + 2 * G * (D + DV) + H * DV) * 2
        return Case(fn, rot, nbytes, "B", "biased_attn_decode_kernel", keep=keep)
    if what == "rec":
        rot = n_rot(2 * B * RH * RK * RV * 4, 300e6)
        state = [torch.zeros(B, RH, RK, RV, **f32) for _ in range(rot)]
        zb, lower, w = torch.full((RH * RK,), 2.0, **f32), torch.full((RH * RK,), 0.5, **f32), torch.ones(RV, **f32)
        c0 = (H + G) * D + G * DV
        work = torch.empty(ob.gated_recurrence_workspace(T, RH, RK, RV), device="cuda", dtype=torch.uint8)
        g = [ob.GatedRecurrence(BF, RH, RK, RV, p + c0 * 2, p + (c0 + RH * RK) * 2, p + (c0 + 2 * RH * RK) * 2, n_mix, zb.data_ptr(),
                                lower.data_ptr(), w.data_ptr(), 1e-6, RV, state[i].data_ptr(), cat.data_ptr() + H * DV * 2, n_cat, 1.0,
                                work.data_ptr()) for i in range(rot)]
        fn = lambda i: ob.gated_recurrence(g[i], tp, T)
        keep = (mix, cat, cu, hist, off, step, state, zb, lower, w, work)
        if prefill:  # decay and write (a product and a multiply-add), read (a multiply-add) per state element and token
            return Case(fn, rot, 5.0 * T * RH * RK * RV, "flop", "gated_recurrence_scan_kernel", launches=3, keep=keep)
        return Case(fn, rot, 2 * B * RH * RK * RV * 4 + B * RH * (2 * RK + 2 * RV) * 2, "B", "gated_recurrence_step_kernel", keep=keep)
    raise ValueError(f"unknown case {name}")


def make_latent_case(name, torch, m, B, ctx, plain=False) -> Case:
    """The fu_ cases: m as in MODELS, optionally with q_rank, kv_rank, window, gla (heads, key, value), gate_rank, experts, top, eff."""
    prefill = name.startswith("prefill_")
    what = name[name.index("fu_") + 3:]
    W, H, D = m["hidden"], m["head_num"], m["head_size"]
    DV, QR, KR = m.get("value_size", D), m.get("q_rank", 1536), m.get("kv_rank", 512)
    RH, RK, RV = m.get("gla", (W // 512, 256, 512))
    E, TOP, EF, rank = m.get("experts", 32), m.get("top", 4), m.get("eff", m["inter_size"] // 4), m.get("gate_rank", 16)
    window = min(m.get("window", 1024), ctx) if prefill else ctx
    T = B * ctx if prefill else B
    bf, f32, i32 = (dict(device="cuda", dtype=t) for t in (torch.bfloat16, torch.float32, torch.int32))
    rnd = lambda *s: 0.02 * torch.randn(*s, **bf)
    n_rot = lambda nbytes, target=400e6: 2 if prefill else max(2, int(target // nbytes) + 1)
    BF = ob.BF16
    n_gla = RH * (2 * RK + 2 * RV) + 16
    plain_shapes = {"in": (W, n_gla), "uq": (QR, H * D), "out": (H * DV, W), "kv": (KR, H * (D + DV))}
    if what in plain_shapes:
        K, N = plain_shapes[what]
        rot = n_rot(K * N * 2)
        x, w = torch.randn(T, K, **bf), [rnd(K, N) for _ in range(rot)]
        stream = what == "out"
        y = torch.zeros(T, N, **(f32 if stream else bf))
        fn = lambda i: ob.project(BF, x, w[i], None, y, T, N, K, f32=stream, resid=y if stream else None, scale=0.3)
        if prefill:
            return Case(fn, rot, 2.0 * T * N * K, "flop", "gemm_tc_kernel (bf16)", keep=(x, w, y))
        return Case(fn, rot, K * N * 2 + T * K * 2 + T * N * (8 if stream else 2), "B", _projection_kernel(T, False) + " (bf16)", keep=(x, w, y))
    if what in ("absorb", "uv"):
        K, N = (D, KR) if what == "absorb" else (KR, DV)
        rot = n_rot(H * K * N * 2)
        x, w, y = torch.randn(T, H * K, **bf), [rnd(H, K, N) for _ in range(rot)], torch.zeros(T, H * N, **bf)
        g = ob.RowGroups(n=H, w_stride=K * N, x_stride=K, y_stride=N)
        fn = lambda i: ob.project(BF, x, w[i], None, y, T, N, K, ldx=H * K, ldy=H * N, ldw=N, groups=g)
        return Case(fn, rot, H * K * N * 2 + T * H * (K + N) * 2, "B", "skinny_kn_staged_kernel (row groups)", keep=(x, w, y, g))
    if what == "norm":
        rows = 4096
        xs = [torch.randn(rows, W, **f32) for _ in range(3)]
        add = [torch.randn(rows * TOP, W, **bf) for _ in range(3)]
        pick = torch.randperm(rows * TOP, device="cuda").to(torch.int32)
        w1, o1 = torch.ones(W, **f32), torch.empty(rows, W, **bf)
        fn = lambda i: ob.norm_rows(BF, xs[i], None, rows, w1, None, o1, None, 1e-6, W, W, add=add[i], add_rows=pick, add_n=TOP, add_scale=0.3)
        return Case(fn, 3, rows * W * (8 + 2 + 2 * TOP), "B", "norm_rows_kernel", keep=(xs, add, pick, w1, o1))
    if what in ("route", "egate", "edown"):
        n = T * TOP
        h, router = torch.randn(T, W, **bf), rnd(W, E)
        z = torch.zeros(T, E, **f32)
        tiles = ob.route_max_tiles(T, E, TOP)
        a = {k: torch.zeros(s, **i32) for k, s in (("slot", n), ("slot_token", n), ("off", E + 1), ("used", E), ("n_used", 1), ("tile_group", tiles),
                                                   ("tile_row", tiles), ("n_tiles", 1), ("choice", n), ("count", E))}
        a.update(slot_weight=torch.zeros(n, **f32), choice_weight=torch.zeros(n, **f32))
        p = {k: v.data_ptr() for k, v in a.items()}
        xs = torch.zeros(n, W, **bf) if T > 64 else None
        r = ob.Route(T, E, TOP, z.data_ptr(), E, dtype=BF, **p)
        if xs is not None:
            r.x, r.xs, r.ld_x = h.data_ptr(), xs.data_ptr(), W

        def choose(i):
            ob.project(BF, h, router, None, z, T, E, W, f32=True)
            ob.route(r)
        keep = (h, router, z, a, xs, r)
        if what == "route":
            nbytes = T * W * 2 + W * E * 2 + T * E * 8 + (T * W * 2 + n * W * 2 if prefill else 0)
            return Case(choose, 2, nbytes, "B", "router projection, route kernels", launches=5 if T > 64 else 2, keep=keep)
        choose(0)
        used = int(a["n_used"].item())
        K, N = (W, EF) if what == "egate" else (EF, W)
        dual = what == "egate"
        rot = n_rot(used * K * N * 2 * (2 if dual else 1))
        w = [rnd(E, K, N) for _ in range(rot)]
        wu = [rnd(E, K, N) for _ in range(rot)] if dual else [None] * rot
        tiled = T > 64
        x = (xs if tiled else h) if dual else torch.randn(n, K, **bf)
        y = torch.zeros(n, N, **bf)
        g = ob.RowGroups(n=E if tiled else min(E, n), used=None if tiled else p["used"], n_used=None if tiled else p["n_used"], off=p["off"],
                         x_rows=p["slot_token"] if dual and not tiled else None, row_scale=p["slot_weight"] if dual else None, w_stride=K * N,
                         tile_group=p["tile_group"], tile_row=p["tile_row"], n_tiles=p["n_tiles"], max_tiles=tiles, weights=E, rows=n)
        fn = lambda i: ob.project(BF, x, w[i], wu[i], y, T, N, K, act=ob.GATE_CLAMPED, limit=7.0, groups=g)
        keep += (w, wu, x, y, g)
        if prefill:
            return Case(fn, rot, 2.0 * n * N * K * (2 if dual else 1), "flop", "gemm_tc_kernel (row groups)", keep=keep)
        return Case(fn, rot, used * K * N * 2 * (2 if dual else 1) + n * (K + N) * 2, "B", "skinny_kn_staged_kernel (row groups)", keep=keep)
    cu = torch.arange(0, B + 1, **i32) * ctx
    hist, off = torch.zeros(B, **i32), torch.zeros(B, **i32)
    step = torch.full((1,), ctx + 1, **i32)
    tp = ob.TokenPositions(cu.data_ptr(), hist.data_ptr(), B, None, None) if prefill else \
        ob.TokenPositions(None, None, B, step.data_ptr(), off.data_ptr())
    if what == "attn" and prefill:
        q, gate, out = torch.randn(T, H * D, **bf), torch.randn(T, H, **bf), torch.zeros(T, H * DV, **bf)
        kv = [torch.randn(T, H * (D + DV), **bf) for _ in range(2)]
        a = [ob.WindowAttn(H, D, DV, window, q.data_ptr(), H * D, kv[i].data_ptr(), H * (D + DV), T, D ** -0.5, gate.data_ptr(), H, out.data_ptr(),
                           H * DV, 1.0) for i in range(2)]
        fn = lambda i: ob.window_attn(a[i], tp, ctx)
        keys = window * (window + 1) / 2 + (ctx - window) * window
        return Case(fn, 2, float(B * H * 2 * (D + DV) * keys), "flop", "biased_attn_tc_kernel<windowed>", keep=(q, gate, out, kv, cu, hist))
    if what == "attn":
        rot = n_rot(B * window * KR * 2, 300e6)
        ring = [torch.randn(B, window, KR, **bf) for _ in range(rot)]
        q, gate, out = torch.randn(B, H, KR, **bf), torch.randn(B, H, **bf), torch.zeros(B, H, KR, **bf)
        ws = torch.empty(ob.latent_attn_workspace(B, H, KR), device="cuda", dtype=torch.uint8)
        a = [ob.LatentAttn(BF, H, KR, window, window, ring[i].data_ptr(), None, 0, None, None, 0, None, None, 0, 0, None, 1e-6, q.data_ptr(),
                           KR ** -0.5, gate.data_ptr(), H, out.data_ptr(), 1.0) for i in range(rot)]
        fn = lambda i: ob.latent_attn(a[i], tp, B, window, ws, plain)
        return Case(fn, rot, B * window * KR * 2 + 2 * B * H * KR * 2, "B", "latent_attn_kernel", launches=2, keep=(ring, q, gate, out, ws, step, off))
    if what == "rec":
        rot = n_rot(2 * B * RH * RK * RV * 4, 300e6)
        state = [torch.zeros(B, RH, RK, RV, **f32) for _ in range(rot)]
        row, out = torch.randn(T, n_gla, **bf), torch.zeros(T, RH * RV, **bf)
        A, zb, w = torch.randn(RH * RK, rank, **f32), torch.full((RH * RK,), 2.0, **f32), torch.ones(RV, **f32)
        work = torch.empty(ob.gated_recurrence_workspace(T, RH, RK, RV, ob.GR_KEYED), device="cuda", dtype=torch.uint8)
        p = row.data_ptr()
        g = [ob.GatedRecurrence(BF, RH, RK, RV, q=p, v=p + 2 * RH * RK * 2, ld=n_gla, zb=zb.data_ptr(), w=w.data_ptr(), eps=1e-6, norm_width=RV,
                                state=state[i].data_ptr(), out=out.data_ptr(), out_ld=RH * RV, out_scale=1.0, work=work.data_ptr(), kind=ob.GR_KEYED,
                                k=p + RH * RK * 2, r=p + RH * (2 * RK + 2 * RV) * 2, rank=rank, A=A.data_ptr(), inv_tau=1 / 16, q_scale=RK ** -0.5,
                                g=p + RH * (2 * RK + RV) * 2) for i in range(rot)]
        fn = lambda i: ob.gated_recurrence(g[i], tp, T)
        keep = (state, row, out, A, zb, w, work, cu, hist, off, step)
        if prefill:  # decay, write and read of a state element and token, as counted for fv_rec
            return Case(fn, rot, 5.0 * T * RH * RK * RV, "flop", "gated_recurrence_scan_kernel", launches=3, keep=keep)
        return Case(fn, rot, 2 * B * RH * RK * RV * 4 + B * RH * (2 * RK + 3 * RV) * 2, "B", "gated_recurrence_step_kernel", keep=keep)
    raise ValueError(f"unknown case {name}")


def make_case(name, torch, model="7b", batch=8, ctx=2040, tp=1, plain=False) -> Case:
    m = MODELS[model] if isinstance(model, str) else model
    if "fu_" in name:
        return make_latent_case(name, torch, m, batch, ctx, plain)
    if "fv_" in name:
        return make_mechanism_case(name, torch, m, batch, ctx, plain)
    HID, D, V = m["hidden"], m["head_size"], m["vocab_size"]
    H, INTER = m["head_num"] // tp, m["inter_size"] // tp
    B = batch
    F16 = ob.F16
    half = dict(device="cuda", dtype=torch.float16)
    rnd = lambda *s: (0.02 * torch.randn(*s, device="cuda")).half()
    act = lambda *s: torch.randn(*s, device="cuda").half()
    n_rot = lambda nbytes, target=400e6: max(2, int(target // nbytes) + 1)

    if name in ("qkv", "gate_up"):
        N = 3 * H * D if name == "qkv" else INTER
        dual = name == "gate_up"
        rot = n_rot(HID * N * 2 * (2 if dual else 1))
        x, w = act(B, HID), [rnd(HID, N) for _ in range(rot)]
        wu = [rnd(HID, N) for _ in range(rot)] if dual else [None] * rot
        out = torch.empty(B, N, **half)
        if plain and dual:
            fn = lambda i: ob.gemm_swiglu(F16, x, w[i], wu[i], out, B, N, HID)
        elif plain:
            fn = lambda i: ob.gemm(F16, x, w[i], out, B, N, HID, ob.W_KN)
        else:  # as in the decode step: raw residual stream in, scaled by rsqrt(mean(x^2) + eps) on the way out
            fn = lambda i: ob.gemm_fused(F16, x, w[i], wu[i], out, B, N, HID, 1e-5, None, None)
        nbytes = (2 if dual else 1) * HID * N * 2 + B * HID * 2 + B * N * 2
        kern = _projection_kernel(B, dual)
        return Case(fn, rot, nbytes, "B", kern, keep=(x, w, wu, out))
    if name in ("o_proj", "down"):
        K = H * D if name == "o_proj" else INTER
        rot = n_rot(K * HID * 2)
        x, w = act(B, K), [rnd(K, HID) for _ in range(rot)]
        res = act(B, HID)
        out = torch.empty(B, HID, **half)
        if plain:
            fn = lambda i: ob.gemm(F16, x, w[i], out, B, HID, K, ob.W_KN)
        else:  # as in the decode step: the result is added to the residual stream in the epilogue
            fn = lambda i: ob.gemm_fused(F16, x, w[i], None, res, B, HID, K, -1.0, res, None)
        nbytes = K * HID * 2 + B * K * 2 + (1 if plain else 2) * B * HID * 2
        return Case(fn, rot, nbytes, "B", _projection_kernel(B, False), keep=(x, w, res, out))
    if name in ("lm_head", "lm_head_kn"):
        lay = ob.W_NK if name == "lm_head" else ob.W_KN
        rot = 2
        x = act(B, HID)
        w = [rnd(V, HID) if lay == ob.W_NK else rnd(HID, V) for _ in range(rot)]
        out = torch.empty(B, V, **half)
        fn = lambda i: ob.gemm(F16, x, w[i], out, B, V, HID, lay)
        kern = "skinny_nk_kernel" if lay == ob.W_NK else _projection_kernel(B, False)
        return Case(fn, rot, V * HID * 2 + B * HID * 2 + B * V * 2, "B", kern, keep=(x, w, out))
    if name == "attn":
        S = ctx + 8
        rot = n_rot(2 * B * H * S * D * 2, 300e6)
        kc = [torch.randn(B, H, S, D, **half) for _ in range(rot)]
        vc = [torch.randn(B, H, S, D, **half) for _ in range(rot)]
        qkv = torch.randn(B, 3 * H, D, **half)
        o = torch.empty(B, H, D, **half)
        wsb = ob.decode_attn_workspace_bytes(B, H, D, S)
        ws = torch.empty(wsb, device="cuda", dtype=torch.uint8)
        p, step = qkv.data_ptr(), ctx + 1
        tickets = torch.zeros(B * H, device="cuda", dtype=torch.int32)
        fn = lambda i: ob.decode_attn(F16, p, p + H * D * 2, p + 2 * H * D * 2, 3 * H * D, 3 * H * D, 3 * H * D, None, None, None,
                                      kc[i], vc[i], H * S * D, S * D, D, B, H, H, D, step, step - 1, D, 10000.0, D ** -0.5, o,
                                      H * D, ws, wsb)
        if plain:  # the one-launch form (splits merged by the last block), which the model class does not use
            fn = lambda i: ob.decode_attn_merged(F16, p, p + H * D * 2, p + 2 * H * D * 2, 3 * H * D, 3 * H * D, 3 * H * D, None,
                                                 None, None, kc[i], vc[i], H * S * D, S * D, D, B, H, H, D, step, None, step - 1, D,
                                                 10000.0, D ** -0.5, o, H * D, ws, wsb, tickets)
        return Case(fn, rot, 2 * ctx * B * H * D * 2 + 5 * B * H * D * 2, "B", "decode_attn_mma_kernel<128,1>",
                    keep=(kc, vc, qkv, o, ws, tickets))
    if name == "attn_c1":
        # the reference's unit-test shape in fp32: 16.9 MB per launch, far below L2 -> rotate over > 126 MB of caches
        Bc, Hc, Dc, Sc, step = 2, 32, 128, 256, 255
        rot = 10
        f32 = dict(device="cuda", dtype=torch.float32)
        kc = [torch.rand(Bc, Hc, Sc, Dc, **f32) * 2 - 1 for _ in range(rot)]
        vc = [torch.rand(Bc, Hc, Sc, Dc, **f32) * 2 - 1 for _ in range(rot)]
        qkv = torch.rand(Bc, 3 * Hc, Dc, **f32) * 2 - 1
        o = torch.empty(Bc, Hc, Dc, **f32)
        wsb = ob.decode_attn_workspace_bytes(Bc, Hc, Dc, Sc)
        ws = torch.empty(wsb, device="cuda", dtype=torch.uint8)
        p = qkv.data_ptr()
        fn = lambda i: ob.decode_attn(ob.F32, p, p + Hc * Dc * 4, p + 2 * Hc * Dc * 4, 3 * Hc * Dc, 3 * Hc * Dc, 3 * Hc * Dc, None,
                                      None, None, kc[i], vc[i], Hc * Sc * Dc, Sc * Dc, Dc, Bc, Hc, Hc, Dc, step, step, Dc, 10000.0,
                                      Dc ** -0.5, o, Hc * Dc, ws, wsb)
        return Case(fn, rot, 2 * (step - 1) * Bc * Hc * Dc * 4 + 245760, "B", "decode_attn_kernel<float,128>", keep=(kc, vc, qkv, o, ws))
    if name in ("norm", "rmsnorm", "norm8"):
        T = B if name == "norm8" else 4096
        rot = 4
        xs, rs = [act(T, HID) for _ in range(rot)], [act(T, HID) for _ in range(rot)]
        g = (1 + 0.1 * torch.randn(HID, device="cuda")).half()
        if name == "rmsnorm":
            fn = lambda i: ob.rmsnorm(F16, xs[i], g, 1e-5, T, HID)
            nbytes = 2 * T * HID * 2 + HID * 2
        else:
            fn = lambda i: ob.add_residual_rmsnorm(F16, rs[i], xs[i], None, g, 1e-5, T, HID)
            nbytes = 4 * T * HID * 2 + 2 * HID * 2
        return Case(fn, rot, nbytes, "B", "rmsnorm_kernel", keep=(xs, rs, g))
    if name in ("topk", "sample"):
        rot = 4
        lg = [torch.randn(B, V, **half) for _ in range(rot)]
        val = torch.empty(B, 64, device="cuda", dtype=torch.float32)
        idx = torch.empty(B, 64, device="cuda", dtype=torch.int32)
        if name == "topk":
            fn = lambda i: ob.topk(F16, lg[i], B, V, 50, val, idx)
            return Case(fn, rot, B * V * 2 + B * 50 * 8, "B", "topk_kernel", keep=(lg, val, idx))
        ob.topk(F16, lg[0], B, V, 50, val, idx)
        out = torch.empty(B, device="cuda", dtype=torch.int32)
        fn = lambda i: ob.topk_sample(idx, val, B, 50, 1.0, 7 + i, V, 2, out)
        return Case(fn, rot, B * 50 * 8 + B * 4, "B", "sample_kernel", keep=(lg, val, idx, out))

    if name == "decode_layer":
        S = ctx + 8
        rot = 2
        w_qkv, w_o = [rnd(HID, 3 * H * D) for _ in range(rot)], [rnd(H * D, HID) for _ in range(rot)]
        w_g, w_u, w_d = [rnd(HID, INTER) for _ in range(rot)], [rnd(HID, INTER) for _ in range(rot)], [rnd(INTER, HID) for _ in range(rot)]
        kc = [torch.randn(B, H, S, D, **half) for _ in range(rot)]
        vc = [torch.randn(B, H, S, D, **half) for _ in range(rot)]
        res, qkv = act(B, HID), torch.empty(B, 3 * H, D, **half)
        o, a = torch.empty(B, H * D, **half), torch.empty(B, INTER, **half)
        wsb = ob.decode_attn_workspace_bytes(B, H, D, S)
        ws = torch.empty(wsb, device="cuda", dtype=torch.uint8)
        p, step = qkv.data_ptr(), ctx + 1

        def fn(i):
            ob.gemm_fused(F16, res, w_qkv[i], None, qkv, B, 3 * H * D, HID, 1e-5, None, None)
            ob.decode_attn(F16, p, p + H * D * 2, p + 2 * H * D * 2, 3 * H * D, 3 * H * D, 3 * H * D, None, None, None, kc[i], vc[i],
                           H * S * D, S * D, D, B, H, H, D, step, step - 1, D, 10000.0, D ** -0.5, o, H * D, ws, wsb)
            ob.gemm_fused(F16, o, w_o[i], None, res, B, HID, H * D, -1.0, res, None)
            ob.gemm_fused(F16, res, w_g[i], w_u[i], a, B, INTER, HID, 1e-5, None, None)
            ob.gemm_fused(F16, a, w_d[i], None, res, B, HID, INTER, -1.0, res, None)

        nbytes = (HID * 3 * H * D + H * D * HID + 3 * HID * INTER) * 2 + 2 * ctx * B * H * D * 2
        return Case(fn, rot, nbytes, "B", "skinny_kn_staged_kernel + decode_attn_mma_kernel", launches=5,
                    keep=(w_qkv, w_o, w_g, w_u, w_d, kc, vc, res, qkv, o, a, ws))

    # ---- context phase: --batch sequences of --ctx new tokens each ---------------------------------------
    P = ctx
    T = B * P
    if name in ("prefill_qkv", "prefill_o", "prefill_gate", "prefill_down", "prefill_lm"):
        K, N, lay = {"prefill_qkv": (HID, 3 * H * D, ob.W_KN), "prefill_o": (H * D, HID, ob.W_KN), "prefill_gate": (HID, INTER, ob.W_KN),
                     "prefill_down": (INTER, HID, ob.W_KN), "prefill_lm": (HID, V, ob.W_KN)}[name]
        rot = 2
        x = act(T, K)
        w = [rnd(K, N) for _ in range(rot)]
        out = torch.empty(T, N, **half)
        if name == "prefill_gate":
            wu = [rnd(K, N) for _ in range(rot)]
            fn = lambda i: ob.gemm_swiglu(F16, x, w[i], wu[i], out, T, N, K)
            return Case(fn, rot, 4.0 * T * N * K, "flop", "gemm_tc_kernel<2>", keep=(x, w, wu, out))
        fn = lambda i: ob.gemm(F16, x, w[i], out, T, N, K, lay)
        return Case(fn, rot, 2.0 * T * N * K, "flop", "gemm_tc_kernel<0>", keep=(x, w, out))
    S = max(2048, P)
    cu = torch.arange(0, B + 1, device="cuda", dtype=torch.int32) * P
    hl = torch.zeros(B, device="cuda", dtype=torch.int32)
    if name == "prefill_attn":
        rot = 2
        q = torch.randn(T, 3 * H * D, **half)
        kc = [torch.randn(B, H, S, D, **half) for _ in range(rot)]
        vc = [torch.randn(B, H, S, D, **half) for _ in range(rot)]
        out = torch.empty(T, H * D, **half)
        fn = lambda i: ob.context_attn(F16, q, 3 * H * D, kc[i], vc[i], H * S * D, S * D, D, cu, hl, B, P, H, H, D, D ** -0.5, out)
        return Case(fn, rot, float(B * H * 4 * D * P * (P + 1) / 2), "flop", "context_attn_tc_kernel", keep=(q, kc, vc, out, cu, hl))
    if name == "prefill_rope":
        rot = 3
        q = [torch.randn(T, 3 * H * D, **half) for _ in range(rot)]
        kc, vc = torch.zeros(B, H, S, D, **half), torch.zeros(B, H, S, D, **half)
        flag = torch.zeros(1, device="cuda", dtype=torch.int32)
        fn = lambda i: ob.qkv_bias_rope_kvcache(F16, q[i], None, cu, hl, kc, vc, H * S * D, S * D, D, T, B, H, H, D, D, 10000.0, S, flag)
        # reads the packed rows, writes q and k back in place and k, v into the cache
        return Case(fn, rot, T * 3 * H * D * 2 + T * 2 * H * D * 2 + T * 2 * H * D * 2, "B", "qkv_rope_kvcache_vec_kernel",
                    keep=(q, kc, vc, flag, cu, hl))
    if name == "prefill_layer":
        rot = 2
        w_qkv, w_o = [rnd(HID, 3 * H * D) for _ in range(rot)], [rnd(H * D, HID) for _ in range(rot)]
        w_g, w_u, w_d = [rnd(HID, INTER) for _ in range(rot)], [rnd(HID, INTER) for _ in range(rot)], [rnd(INTER, HID) for _ in range(rot)]
        g = torch.ones(HID, **half)
        x0 = act(T, HID)
        y, res = torch.empty(T, HID, **half), torch.zeros(T, HID, **half)
        qkv, attn, a = torch.empty(T, 3 * H * D, **half), torch.empty(T, H * D, **half), torch.empty(T, INTER, **half)
        kc, vc = torch.zeros(B, H, S, D, **half), torch.zeros(B, H, S, D, **half)
        flag = torch.zeros(1, device="cuda", dtype=torch.int32)

        n_parts = ob.gemm_rows_parts(HID)
        ss_a = torch.ones(T, n_parts, device="cuda", dtype=torch.float32)
        ss_b = torch.ones(T, n_parts, device="cuda", dtype=torch.float32)

        def fn(i):
            # one layer of the context phase as the model runs it on one GPU: what LlamaContextDecoder::forward does per layer
            # (src/layers/decoder/context_decoder.cpp:95-131) without norm kernels -- the projections behind a norm scale their
            # rows from the statistics the projection before them left, o_proj and down_proj add into the residual stream
            ob.gemm_rows(F16, res, w_qkv[i], None, qkv, T, 3 * H * D, HID, row_ss=ss_a, ss_parts=n_parts)
            ob.qkv_bias_rope_kvcache(F16, qkv, None, cu, hl, kc, vc, H * S * D, S * D, D, T, B, H, H, D, D, 10000.0, S, flag)
            ob.context_attn(F16, qkv, 3 * H * D, kc, vc, H * S * D, S * D, D, cu, hl, B, P, H, H, D, D ** -0.5, attn)
            ob.gemm_rows(F16, attn, w_o[i], None, res, T, HID, H * D, resid=res, row_ss_out=ss_b)
            ob.gemm_rows(F16, res, w_g[i], w_u[i], a, T, INTER, HID, row_ss=ss_b, ss_parts=n_parts)
            ob.gemm_rows(F16, a, w_d[i], None, res, T, HID, INTER, resid=res, row_ss_out=ss_a)

        # dense flops: projections + both attention products over the full square (the causal half is skipped)
        flops = 2.0 * T * HID * (3 * H * D + H * D) + 6.0 * T * HID * INTER + 4.0 * B * H * D * P * P
        return Case(fn, rot, flops, "flop", "gemm_tc_kernel", launches=6,
                    keep=(w_qkv, w_o, w_g, w_u, w_d, g, x0, y, res, qkv, attn, a, kc, vc, flag, cu, hl, ss_a, ss_b))
    raise ValueError(f"unknown case {name}")


def time_case(case: Case, torch, iters=20, warm=5, graph=False) -> float:
    """Mean seconds per call of case.fn: CUDA events on the launching stream, after warm-up, rotating buffers."""
    st = torch.cuda.current_stream()
    for i in range(warm):
        case.fn(i % case.rot)
    st.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if graph:
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for i in range(iters):
                case.fn(i % case.rot)
        g.replay()
        torch.cuda.synchronize()
        e0.record()
        g.replay()
        e1.record()
        torch.cuda.synchronize()
    else:
        e0.record(st)
        for i in range(iters):
            case.fn(i % case.rot)
        e1.record(st)
        st.synchronize()
    return e0.elapsed_time(e1) / iters * 1e-3


def main():
    import torch
    ap = argparse.ArgumentParser()
    ap.add_argument("case", choices=DECODE_CASES + PREFILL_CASES)
    ap.add_argument("--model", default="7b", choices=sorted(MODELS))
    ap.add_argument("--iters", type=int, default=6)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--ctx", type=int, default=None, help="cache rows (decode cases, default 2040) / new tokens per sequence (prefill cases, default 512)")
    ap.add_argument("--graph", action="store_true", help="time a CUDA graph of the launches (device-side back-to-back)")
    ap.add_argument("--tp", type=int, default=1, help="per-rank shapes of a tensor-parallel degree (heads and FFN columns divided)")
    ap.add_argument("--plain", action="store_true", help="projections through onellm_gemm / onellm_gemm_swiglu instead of onellm_gemm_fused; attn: onellm_decode_attn_merged (splits merged inside the kernel) instead of onellm_decode_attn")
    a = ap.parse_args()
    ctx = a.ctx if a.ctx is not None else (512 if a.case.startswith("prefill_") else 2040)
    torch.cuda.set_device(0)
    torch.manual_seed(0)
    case = make_case(a.case, torch, a.model, a.batch, ctx, a.tp, a.plain)
    t = time_case(case, torch, iters=a.iters, warm=3, graph=a.graph)
    flag = ob.lib().onellm_gemm_timeout_flag()
    if case.unit == "flop":
        print(f"{a.case}: {t * 1e6:.1f} us/call, {case.amount / t / 1e12:.0f} TFLOP/s ({case.amount:.0f} flops, {case.launches} launch(es)), "
              f"time-out flag {flag}")
    else:
        print(f"{a.case}: {t * 1e6:.1f} us/launch, {case.amount / t / 1e9:.0f} GB/s algorithmic ({int(case.amount)} bytes), kernel {case.kernel}")


if __name__ == "__main__":
    main()
