"""Timing of the unquantized designs at equal size (``bench.py --design``): Zokunex beside the quantized decoder, Femirax
beside Zokunex.

Every figure is a device time (CUDA events) over launches captured in a CUDA graph whose inputs rotate over more memory
than the L2 cache holds; weights are random.  A kernel's roofline is the slower of its algorithmic bytes at the measured
copy bandwidth and its algorithmic FLOPs at the measured bf16 product rate.
"""

from __future__ import annotations

import torch

from . import _lib, dense, layers, synthetic
from .cache import DecayState, KeyValueState, LatentState, MatrixMemoryState
from .graph_wrapper import GLoRCQGraphWrapper

ROTATE_BYTES = 400e6        # memory the inputs of a timed kernel rotate over (L2: 126 MB)

# width, dense ff, experts, top, expert ff, mLSTM (heads, dim, vdim), latent (heads, dim, rot, vdim, rank), vocab
SIZES = {
    "small": dict(width=1024, ff=2816, experts=32, identity=2, top=4, eff=704, ml=(4, 128, 256), la=(8, 64, 32, 64, 256), vocab=32000),
    "medium": dict(width=2048, ff=5632, experts=60, identity=4, top=4, eff=1408, ml=(4, 256, 512), la=(16, 128, 64, 128, 512), vocab=151936),
    "large": dict(width=4096, ff=14336, experts=8, identity=1, top=2, eff=14336, ml=(8, 256, 512), la=(32, 128, 64, 128, 512), vocab=32000),
}


def zokunex_config(size, n_layers=8):
    s = SIZES[size]
    H, D, V = s["ml"]
    h, d, r, v, k = s["la"]
    out = []
    for l in range(n_layers):
        mixer = ({"type": "latent_attention", "mixer": {"heads": h, "dim": d, "rot_dim": r, "vdim": v, "kv_rank": k, "scale": (d + r) ** -0.5,
                                                        "rot": {"base": 1e6, "dims": r}}} if l % 4 == 1 else
                 {"type": "mlstm", "mixer": {"heads": H, "dim": D, "vdim": V, "gate_cap": 15.0}})
        mlp = {"kind": "dense", "ff": s["ff"]} if l == 0 else \
            {"kind": "moe", "expert": {"ff": s["eff"]}, "router": {"experts": s["experts"], "identity": s["identity"], "top": s["top"]}}
        out.append(dict(mixer, mlp=mlp))
    return {"architecture": "Zokunex", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": out}


def closest_config(size, n_layers=8):
    """The quantized decoder's shape of equal width, depth, experts and vocabulary (a softmax top-k block with SwiGLU experts)."""
    s = SIZES[size]
    heads = s["width"] // 128
    return dict(hidden_size=s["width"], num_hidden_layers=n_layers, num_attention_heads=heads, num_key_value_heads=heads,
                vocab_size=s["vocab"], num_experts=s["experts"], num_experts_per_tok=s["top"], moe_intermediate_size=s["eff"],
                shared_expert_intermediate_size=s["ff"], norm_topk_prob=False, rms_norm_eps=1e-6, rope_theta=1e6,
                max_position_embeddings=8192)


# Femirax: width, ff, retention (heads, dim, vdim), attention (heads, key heads, dim), linear attention (heads, dim, vdim),
# token side
FEMIRAX_SIZES = {
    "small": dict(ret=(4, 128, 256), att=(8, 2, 128), gla=(4, 128, 256), side=128, ff=1408),
    "medium": dict(ret=(4, 256, 512), att=(16, 4, 128), gla=(4, 256, 512), side=256, ff=2816),
    "large": dict(ret=(8, 256, 512), att=(32, 8, 128), gla=(8, 256, 512), side=256, ff=14336),
}


def femirax_config(size, n_layers=8):
    s, f = SIZES[size], FEMIRAX_SIZES[size]
    out = []
    for l in range(n_layers):
        H, D, V = f["ret"]
        if l % 4 == 1:
            h, kv, d = f["att"]
            gh, gd, gv = f["gla"]
            mixer = {"type": "parallel", "mixer": {"left": {"heads": h, "kv_heads": kv, "dim": d, "vdim": d, "scale": d ** -0.5,
                                                            "rot": {"base": 1e6, "dims": d}},
                                                   "right": {"heads": gh, "dim": gd, "vdim": gv, "tau": 16.0}}}
        else:
            mixer = {"type": "retention", "mixer": {"heads": H, "dim": D, "vdim": V, "decay": [1 - 2.0 ** (-5 - i) for i in range(H)],
                                                    "rot": {"base": 1e6, "dims": D}}}
        out.append(dict(mixer, mlp={"kind": "dense", "ff": f["ff"]}))
    return {"architecture": "Femirax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "token_side": {"dim": f["side"]}, "layers": out}


def zokunex_beside_femirax(size, n_layers=8):
    """Zokunex with a dense feed-forward of as many weights in every layer."""
    cfg = zokunex_config(size, n_layers)
    return dict(cfg, layers=[dict(L, mlp={"kind": "dense", "ff": FEMIRAX_SIZES[size]["ff"] * 3 // 2}) for L in cfg["layers"]])


def graph_time(fns, reps=5):
    """Seconds per call of a list of closures, captured back to back into one graph: best of ``reps`` replays."""
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        for f in fns[:2]:
            f()
    torch.cuda.current_stream().wait_stream(s)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=s):
        for f in fns:
            f()
    for _ in range(3):
        g.replay()
    times = []
    for _ in range(reps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        g.replay()
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1) * 1e-3 / len(fns))
    return min(times)


def event_time(fn, reps=5):
    for _ in range(3):
        fn()
    times = []
    for _ in range(reps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1) * 1e-3)
    return min(times)


class Table:
    def __init__(self, gbs, tflops):
        self.gbs, self.tflops, self.rows = gbs, tflops, []

    def add(self, name, sec, nbytes=0.0, flops=0.0, like=None):
        bound = max(nbytes / (self.gbs * 1e9), flops / (self.tflops * 1e12))
        self.rows.append({"kernel": name, "us": round(sec * 1e6, 2), "roofline_us": round(bound * 1e6, 2), "frac": round(bound / sec, 3),
                          "bound": "hbm" if nbytes / (self.gbs * 1e9) >= flops / (self.tflops * 1e12) else "tensor",
                          **({"like": like} if like else {})})


def _copies(nbytes):
    return max(1, min(64, int(ROTATE_BYTES // max(nbytes, 1)) + 1))


def decode_kernels(t, size, context, batch=1):
    dev, bf = torch.device("cuda:0"), torch.bfloat16
    s = SIZES[size]
    C, B = s["width"], batch

    def product(name, rows, N, K, split, **kw):
        n = _copies(2 * N * K)
        W = [torch.randn(N, K, device=dev).mul_(K ** -0.5).to(bf) for _ in range(n)]
        x = torch.randn(rows, K, device=dev).to(bf)
        sec = graph_time([lambda w=w: dense.matmul(x, w, split=split, **kw) for w in W])
        t.add(f"{name} ({rows} x {N} x {K})", sec, 2 * N * K, 2.0 * rows * N * K, "output projection")
    H, D, V = s["ml"]
    product("product: q k v gates", B, 2 * H * (D + V) + 2 * H, C, 2 * H * (D + V))
    product("product: mLSTM output", B, C, H * V, 0)
    product("product: dense up, relu^2", B, s["ff"], C, s["ff"], act=layers.ACTIVATIONS["relu2"])
    product("product: dense down", B, C, s["ff"], 0)

    E, top, ff = s["experts"], s["top"], s["eff"]
    n = min(_copies(2 * E * ff * C), 4)
    ups, downs = [torch.randn(E, ff, C, device=dev).to(bf) for _ in range(n)], [torch.randn(E, C, ff, device=dev).to(bf) for _ in range(n)]
    h, mid = torch.randn(B, C, device=dev).to(bf), torch.randn(B * top, ff, device=dev).to(bf)
    plans = [dense.route(torch.randn(B, E, device=dev), torch.zeros(E, device=dev), E, 0, top) for _ in range(16)]
    live = sum(int(p.sel.unique().numel()) for p in plans) / len(plans)
    sec = graph_time([lambda p=p, i=i: dense.matmul(h, ups[i % n], plan=p, act=layers.ACTIVATIONS["gelu_erf"]) for i, p in enumerate(plans)])
    t.add(f"experts up, gelu ({live:.1f} of {E}, {ff} x {C})", sec, live * 2 * ff * C, 0, "expert block")
    sec = graph_time([lambda p=p, i=i: dense.matmul(mid, downs[i % n], plan=p, gathered=False) for i, p in enumerate(plans)])
    t.add(f"experts down ({live:.1f} of {E}, {C} x {ff})", sec, live * 2 * ff * C, 0, "expert block")
    logits, corr = torch.randn(B, E + s["identity"], device=dev), torch.zeros(E + s["identity"], device=dev)
    sec = graph_time([lambda: dense.route(logits, corr, E, s["identity"], top)] * 20)
    t.add("routing and lists", sec, 0, 0, "expert block")

    n = _copies(B * H * D * V * 4)
    states = [MatrixMemoryState(B, H, D, V, dev) for _ in range(n)]
    qkvg, gates = torch.randn(B, 2 * H * (D + V), device=dev).to(bf), torch.randn(B, 2 * H, device=dev)
    one, bias = torch.ones(H * V, device=dev), torch.zeros(H, device=dev)
    sec = graph_time([lambda st=st: dense.mlstm(qkvg, gates, B, 1, H, D, V, 15.0, 1e-5, bias, bias, one, st, False, True, True) for st in states])
    t.add(f"mLSTM step ({B} x {H} heads, {D} x {V})", sec, B * H * D * V * 8, 0, "decode attention")

    hh, d, r, v, k = s["la"]
    n = _copies(B * context * (k + r) * 2)
    caches = [LatentState(B, context, k, r, dev, bf) for _ in range(n)]
    for c in caches:
        c.rows.normal_()
    ukt, uv = torch.randn(hh, k, d, device=dev).to(bf), torch.randn(hh * v, k, device=dev).to(bf)
    start = torch.tensor([context - 1], device=dev)
    cos, sin = layers.rotation_tables(r, context, 1e6, dev)
    q, rest = torch.randn(B, hh * (d + r), device=dev).to(bf), torch.randn(B, k + r + hh, device=dev)
    nw, y = torch.ones(k, device=dev), torch.empty(B, hh * v, device=dev, dtype=bf)

    def call(c):
        return dense.Latent(q, rest, rest[:, k + r:], start, B, 1, hh, d, r, v, k, r, (d + r) ** -0.5, 1e-5, nw, cos, sin, c, y)
    sec = graph_time([lambda c=c: call(c).absorbed(ukt, uv) for c in caches])
    t.add(f"latent attention, absorbed ({B} x {context} positions, {hh} heads, rank {k})", sec,
          B * context * (k + r) * 2 + hh * k * (d + v) * 2, 2.0 * B * hh * context * (2 * k + r), "decode attention")
    sec = graph_time([lambda c=c: call(c).prep() for c in caches] * 2)
    t.add("latent norm, rotation, cache write", sec, B * (k + r) * 6, 0)
    x, yy, w = torch.randn(B, C, device=dev), torch.randn(B, C, device=dev), torch.ones(C, device=dev)
    sec = graph_time([lambda: dense.add_norm(x, yy, w, 1e-5, bf)] * 20)
    t.add("norm and residual", sec, B * C * 14, 0, "add_rmsnorm")
    Wh = [torch.randn(s["vocab"], C, device=dev).to(bf) for _ in range(_copies(2 * s["vocab"] * C))]
    scratch = {}
    dense.head(h, Wh[0], 1.0, scratch)
    sec = graph_time([lambda w=w: dense.head(h, w, 1.0, scratch) for w in Wh])
    t.add(f"output projection ({B} x {s['vocab']} x {C})", sec, 2 * s["vocab"] * C, 0, "output projection")


def prompt_kernels(t, size, T):
    dev, bf = torch.device("cuda:0"), torch.bfloat16
    s = SIZES[size]
    C = s["width"]

    def product(name, N, K, split, **kw):
        x, W = torch.randn(T, K, device=dev).to(bf), torch.randn(N, K, device=dev).mul_(K ** -0.5).to(bf)
        sec = graph_time([lambda: dense.matmul(x, W, split=split, **kw)] * 6)
        ref = graph_time([lambda: x @ W.T] * 6)
        t.add(f"{name} ({T} x {N} x {K}); library product {ref * 1e6:.1f} us", sec, 2 * (N * K + T * K + T * N), 2.0 * T * N * K, "dequant-GEMM")
    H, D, V = s["ml"]
    product("product: q k v gates", 2 * H * (D + V) + 2 * H, C, 2 * H * (D + V))
    product("product: mLSTM output", C, H * V, 0)
    product("product: dense up, relu^2", s["ff"], C, s["ff"], act=layers.ACTIVATIONS["relu2"])
    product("product: dense down", C, s["ff"], 0)
    hh, d, r, v, k = s["la"]
    product("product: keys and values from latents", hh * (d + v), k, hh * (d + v))

    E, top, ff = s["experts"], s["top"], s["eff"]
    up, down = torch.randn(E, ff, C, device=dev).to(bf), torch.randn(E, C, ff, device=dev).to(bf)
    h, mid = torch.randn(T, C, device=dev).to(bf), torch.randn(T * top, ff, device=dev).to(bf)
    logits, corr = torch.randn(T, E + s["identity"], device=dev), torch.zeros(E + s["identity"], device=dev)
    p = dense.route(logits, corr, E, s["identity"], top)
    ent = int((p.tok_entries >= 0).sum())
    nb = 2 * E * ff * C + 2 * ent * (C + ff)
    sec = graph_time([lambda: dense.matmul(h, up, plan=p, act=layers.ACTIVATIONS["gelu_erf"])] * 4)
    t.add(f"experts up, gelu ({ent} entries, {E} x {ff} x {C})", sec, nb, 2.0 * ent * ff * C, "dequant-GEMM")
    sec = graph_time([lambda: dense.matmul(mid, down, plan=p, gathered=False)] * 4)
    t.add(f"experts down ({ent} entries, {E} x {C} x {ff})", sec, nb, 2.0 * ent * ff * C, "dequant-GEMM")
    sec = graph_time([lambda: dense.route(logits, corr, E, s["identity"], top)] * 4)
    t.add("routing and lists", sec, T * (E + s["identity"]) * 4 + T * top * 24, 0, "expert block")
    x, out, w = torch.randn(T, C, device=dev), torch.randn(T * top, C, device=dev).to(bf), torch.ones(C, device=dev)
    sec = graph_time([lambda: dense.combine_norm(x, out, p, w, 1e-5, bf)] * 4)
    t.add("experts' sum, norm and residual", sec, ent * C * 2 + T * C * 10, 0, "combine")
    yy = torch.randn(T, C, device=dev)
    sec = graph_time([lambda: dense.add_norm(x, yy, w, 1e-5, bf)] * 4)
    t.add("norm and residual", sec, T * C * 14, 0, "add_rmsnorm")

    st = MatrixMemoryState(1, H, D, V, dev)
    qkvg, gates = torch.randn(T, 2 * H * (D + V), device=dev).to(bf), torch.randn(T, 2 * H, device=dev)
    one, bias = torch.ones(H * V, device=dev), torch.full((H,), 3.0, device=dev)
    sec = graph_time([lambda: dense.mlstm(qkvg, gates, 1, T, H, D, V, 15.0, 1e-5, bias, bias, one, st, True)] * 4)
    # per position and head: scores and weighted values inside a block of 64 (half of it visible), state read and update
    t.add(f"mLSTM, blocks ({T} positions, {H} heads, {D} x {V})", sec, T * H * (2 * D + 3 * V) * 2,
          2.0 * T * H * (32 * (D + V) + 2 * D * V), "prompt attention")

    c = LatentState(1, T, k, r, dev, bf)
    c.rows.normal_()
    start = torch.zeros(1, dtype=torch.long, device=dev)
    cos, sin = layers.rotation_tables(r, T, 1e6, dev)
    q, rest = torch.randn(T, hh * (d + r), device=dev).to(bf), torch.randn(T, k + r + hh, device=dev)
    nw, y, kv = torch.ones(k, device=dev), torch.empty(T, hh * v, device=dev, dtype=bf), torch.randn(T, hh * (d + v), device=dev).to(bf)

    def call():
        return dense.Latent(q, rest, rest[:, k + r:], start, 1, T, hh, d, r, v, k, r, (d + r) ** -0.5, 1e-5, nw, cos, sin, c, y)
    vt = torch.randn(hh * v, dense.ceil_to(T, 8), device=dev).to(bf)
    two = call().prefill_form() == 2
    keys = kv[:, :hh * d].contiguous() if two else kv
    sec = graph_time([lambda: call().prefill(keys, T, vt if two else None)] * 4)
    t.add(f"latent attention, prompt ({T} positions, {hh} heads, {d + r} / {v})", sec, T * hh * (2 * d + r + 2 * v) * 2,
          float(T) * T * hh * (d + r + v), "prompt attention")
    sec = graph_time([lambda: call().prep()] * 4)
    t.add("latent norm, rotation, cache write", sec, T * ((k + r) * 6 + hh * r * 4), 0, "rope_prefill")


def like_kernels(t, size, context, T):
    """The quantized decoder's kernels of the same roles."""
    from . import _lib
    import ctypes as C_
    dev, L = torch.device("cuda:0"), _lib.lib()
    s = SIZES[size]
    C = s["width"]
    nh = C // 128
    f16 = torch.float16

    def stream():
        return torch.cuda.current_stream().cuda_stream
    nc = _copies(2 * context * C * 2)
    kc, vc = torch.randn(nc, nh, context, 128, device=dev, dtype=f16), torch.randn(nc, nh, context, 128, device=dev, dtype=f16)
    q = torch.randn(C, device=dev, dtype=f16)
    cs, pos = torch.ones(context, 128, device=dev, dtype=f16), torch.tensor([context - 1], device=dev)
    y = torch.empty_like(q)
    ws = torch.empty(L.glq_attn_decode_workspace_bytes(1, nh, 128, context), dtype=torch.uint8, device=dev)
    ctr = torch.zeros(nh, dtype=torch.int32, device=dev)

    def attn(i):
        _lib.check(L.glq_attn_decode(q.data_ptr(), q.data_ptr(), q.data_ptr(), cs.data_ptr(), cs.data_ptr(), pos.data_ptr(), kc[i].data_ptr(),
                                     vc[i].data_ptr(), y.data_ptr(), 1, nh, nh, 128, context, None, None, 1e-6, ws.data_ptr(), ws.numel(),
                                     ctr.data_ptr(), ctr.numel(), stream()))
    sec = graph_time([lambda i=i: attn(i) for i in range(nc)])
    t.add(f"decode attention ({context} positions, {nh} heads x 128)", sec, 2 * context * C * 2)
    qq = torch.randn(T, C, device=dev, dtype=f16)
    yy = torch.empty_like(qq)
    sec = graph_time([lambda: _lib.check(L.glq_attn_prefill(qq.data_ptr(), qq.data_ptr(), qq.data_ptr(), yy.data_ptr(), 1, T, nh, nh, 128, stream()))] * 4)
    t.add(f"prompt attention ({T} positions, {nh} heads x 128)", sec, 4 * T * C * 2, 2.0 * T * T * C)
    x, w, o1, o2 = torch.randn(T, C, device=dev, dtype=f16), torch.ones(C, device=dev, dtype=f16), torch.empty_like(qq), torch.empty_like(qq)
    for rows in (1, T):
        sec = graph_time([lambda: _lib.check(L.glq_add_rmsnorm(x.data_ptr(), qq.data_ptr(), w.data_ptr(), 1e-6, rows, C, o1.data_ptr(), o2.data_ptr(), stream()))] * 8)
        t.add(f"add_rmsnorm ({rows} rows)", sec, rows * C * 8)
    V = s["vocab"]
    Wh = [torch.randn(V, C, device=dev).half() for _ in range(_copies(2 * V * C))]
    lg, best = torch.empty(1, V, device=dev, dtype=f16), torch.empty(1, dtype=torch.int64, device=dev)
    lws, lctr = torch.empty(L.glq_lm_head_workspace_bytes(), dtype=torch.uint8, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    sec = graph_time([lambda w=w: _lib.check(L.glq_lm_head(x.data_ptr(), C, w.data_ptr(), 1, V, C, lg.data_ptr(), V, best.data_ptr(), lws.data_ptr(),
                                                           lws.numel(), lctr.data_ptr(), stream())) for w in Wh])
    t.add(f"output projection ({V} x {C}, fp16)", sec, 2 * V * C)
    # the quantized expert block (2-bit codes): one token, and a prompt
    from .moe_block import GraphCompatibleMoeBlock
    cfg = {**closest_config(size, 1)}
    model = synthetic.make_decoder(cfg, dev, seed=5)
    blk = model.mlp[0]
    assert isinstance(blk, GraphCompatibleMoeBlock)
    for rows in (1, T):
        hx = torch.randn(1, rows, C, device=dev, dtype=f16)
        sec = graph_time([lambda: blk(hx)] * 4)
        E, I, k, Is = s["experts"], s["eff"], s["top"], s["ff"]
        live = min(E, rows * k)
        t.add(f"expert block, 2-bit ({rows} rows)", sec, live * 3 * C * I * 0.28 + 3 * C * Is * 0.28 + rows * C * 4, 6.0 * rows * C * (k * I + Is))


def _product(t, name, rows, N, K, split, like, **kw):
    dev, bf = torch.device("cuda:0"), torch.bfloat16
    x = torch.randn(rows, K, device=dev).to(bf)
    if rows <= 64:
        W = [torch.randn(N, K, device=dev).mul_(K ** -0.5).to(bf) for _ in range(_copies(2 * N * K))]
        sec, note = graph_time([lambda w=w: dense.matmul(x, w, split=split, **kw) for w in W]), ""
    else:
        W = torch.randn(N, K, device=dev).mul_(K ** -0.5).to(bf)
        sec = graph_time([lambda: dense.matmul(x, W, split=split, **kw)] * 6)
        note = f"; library product {graph_time([lambda: x @ W.T] * 6) * 1e6:.1f} us"
    t.add(f"{name} ({rows} x {N} x {K}{note})", sec, 2.0 * (N * K + rows * K) + rows * (2.0 * split + 4.0 * (N - split)), 2.0 * rows * N * K, like)


def femirax_kernels(t, size, rows, T, context):
    """The kernels of one pass over ``rows`` = sequences * T rows; T = 1: a decode step behind ``context`` positions."""
    dev, bf = torch.device("cuda:0"), torch.bfloat16
    s, f = SIZES[size], FEMIRAX_SIZES[size]
    C, B, decode, ff, E = s["width"], rows // T, T == 1, f["ff"], f["side"]
    H, D, V = f["ret"]
    h, kv, d = f["att"]
    gh, gd, gv = f["gla"]
    silu = _lib.GATE_SILU
    _product(t, "product: retention q k v g", rows, 2 * H * (D + V), C, 2 * H * (D + V), "product: q k v gates")
    w = (h + kv) * d + 2 * gh * (gd + gv)
    _product(t, "product: both sides' q k v g and decay rank", rows, w + 16, C, w, "product: q k v gates")
    _product(t, "product: gate and up, silu", rows, 2 * ff, C, 2 * ff, "product: dense up", act=_lib.ACT_SILU_GLU)
    ids = torch.zeros(rows, dtype=torch.long, device=dev)
    table = torch.randn(64, E, device=dev).to(bf)
    _product(t, "product: token side gate, gelu, row of the table", rows, E, C, E, "product: small", act=_lib.ACT_GELU_TANH, mul=table, mul_row=ids)
    _product(t, "product: token side projection", rows, C, E, 0, "product: small")
    n = _copies(rows * C * 10)
    xs = [torch.randn(rows, C, device=dev) for _ in range(min(n, 16))]
    for name, K in (("feed-forward output", ff), ("retention output", H * V)):
        nw = _copies(2 * C * K) if decode else 1
        Ws = [torch.randn(C, K, device=dev).mul_(K ** -0.5).to(bf) for _ in range(nw)]
        y = torch.randn(rows, K, device=dev).to(bf)
        sec = graph_time([lambda i=i, w=w: dense.matmul_add(y, w, xs[i % len(xs)], True) for i, w in enumerate(Ws * (1 if decode else 6))])
        t.add(f"product added to the residual: {name} ({rows} x {C} x {K})", sec, 2.0 * C * K + rows * (2.0 * K + 10 * C), 2.0 * rows * C * K, "product: output")
    y1, y2, ones = torch.randn(rows, C, device=dev), torch.randn(rows, C, device=dev), torch.ones(C, device=dev)
    sec = graph_time([lambda x=x: dense.rms_add(x, 1e-6, bf, y1, ones, norm_w=ones) for x in xs] * 2)
    t.add(f"norm, residual, next norm ({rows} rows)", sec, rows * C * 14, 0, "norm and residual")
    sec = graph_time([lambda x=x: dense.rms_add(x, 1e-6, bf, y1, ones, y2, ones, 0.5, ones) for x in xs] * 2)
    t.add(f"two norms, mean, residual, next norm ({rows} rows)", sec, rows * C * 18, 0, "norm and residual")

    start = torch.tensor([context - 1 if decode else 0], device=dev)
    for name, (nh, nd, nv) in (("retention", f["ret"]), ("gated linear attention", f["gla"])):
        qkvg, a = torch.randn(rows, 2 * nh * (nd + nv), device=dev).to(bf), torch.randn(rows, 16, device=dev)
        q, k, v, g = qkvg.split([nh * nd, nh * nd, nh * nv, nh * nv], 1)
        kw = dict(decay=torch.tensor([1 - 2.0 ** (-5 - i) for i in range(nh)], device=dev), start=start,
                  rotation=layers.Rotation(nd, 1e6, False)(context + 8, dev), k_scale=nd ** -0.5) if name == "retention" else \
            dict(gates=(a, torch.randn(nh * nd, 16, device=dev).mul_(0.25).to(bf), torch.full((nh * nd,), 4.0, device=dev), 16.0), q_scale=nd ** -0.5)
        nw = None if name == "retention" else torch.ones(nv, device=dev)
        states = [DecayState(B, context + 8, nh, nd, nv, dev) for _ in range(_copies(B * nh * nd * nv * 4) if decode else 4)]
        sec = graph_time([lambda st=st: dense.decay_attention(q, k, v, g, B, T, nh, nd, nv, st, nw, 1e-6, silu, short=decode, **kw)
                          for st in states])
        if decode:
            t.add(f"{name} step with norm and gate ({B} x {nh} heads, {nd} x {nv})", sec, B * nh * nd * nv * 8, 0, "mLSTM step")
        else:
            # per position and head: weights and weighted values inside a block of 64 (half of it visible), state read and update
            t.add(f"{name}, blocks ({T} positions, {nh} heads, {nd} x {nv})", sec, rows * nh * (2 * nd + 3 * nv) * 2,
                  2.0 * rows * nh * (32 * (nd + nv) + 2 * nd * nv), "mLSTM, blocks")

    S = context if decode else T
    caches = [KeyValueState(B, S, kv, d, d, dev, bf) for _ in range(_copies(B * S * kv * d * 4) if decode else 2)]
    for c in caches:
        c.k.normal_()
        c.v.normal_()
    qk = torch.randn(rows, (h + kv) * d, device=dev).to(bf)
    rot = layers.Rotation(d, 1e6, True)(S, dev)
    start = torch.tensor([S - 1 if decode else 0], device=dev)
    sec = graph_time([lambda c=c: dense.gqa(qk[:, :h * d], qk[:, h * d:], qk[:, h * d:], B, T, h, kv, d, d, c, d ** -0.5, 1e-6, start,
                                            None if decode else T, rot, True) for c in caches])
    if decode:
        t.add(f"attention, splits ({B} x {S} positions, {h} heads on {kv}, {d})", sec, B * S * kv * d * 4, 4.0 * B * h * S * d, "latent attention, absorbed")
    else:
        t.add(f"attention with norm, rotation, cache write ({T} positions, {h} heads on {kv}, {d})", sec, rows * (2 * h + 4 * kv) * d * 2,
              2.0 * rows * T * h * d, "latent attention, prompt")


def whole_model(design, size, prompt, steps, batch, n_layers):
    """Decode and prompt rates of the two decoders through the generation wrapper."""
    dev = torch.device("cuda:0")
    out = {}
    for name in ((design, "closest") if design == "zokunex" else (design, "closest (zokunex)")):
        if name == "femirax":
            cfg = femirax_config(size, n_layers)
            model, nbytes = synthetic.make_femirax(cfg, dev, seed=3), synthetic.femirax_bytes_per_token(cfg, prompt, batch)
        elif name != "closest":
            cfg = zokunex_config(size, n_layers) if design == "zokunex" else zokunex_beside_femirax(size, n_layers)
            model, nbytes = synthetic.make_zokunex(cfg, dev, seed=3), synthetic.zokunex_bytes_per_token(cfg, prompt, batch)
        else:
            cfg = closest_config(size, n_layers)
            model = synthetic.make_decoder(cfg, dev, seed=3)
            nbytes = None
        vocab = cfg["vocab_size"] if name == "closest" else cfg["vocab"]
        w = GLoRCQGraphWrapper(model, max_batch_size=batch, max_seq_len=prompt + steps + 16)
        ids = torch.randint(0, vocab, (batch, prompt), generator=torch.Generator().manual_seed(1)).to(dev)
        w.generate(ids, max_new_tokens=4)
        one = ids[:1] if batch > 1 else ids

        def prompt_pass():
            w.static_cache.reset()
            w.model(input_ids=ids, cache_position=torch.arange(prompt, device=dev), past_key_values=w.static_cache, logits_to_keep=1)
        sec_p = event_time(prompt_pass)
        tok = one.new_zeros(batch, 1)

        def window():
            for i in range(steps):
                w.replay(tok, prompt + i)
        sec_d = event_time(window) / steps
        out[name] = {"decode_tok_s": round(batch / sec_d, 1), "decode_us_per_step": round(sec_d * 1e6, 1),
                     "prompt_tok_s": round(batch * prompt / sec_p, 0), "prompt_ms": round(sec_p * 1e3, 2)}
        if nbytes:
            out[name]["decode_bytes_per_step"] = nbytes
        del w, model
        torch.cuda.empty_cache()
    return out


def run(design, size, prompt, steps, batch, n_layers, gbs, tflops, kernels=True):
    line = {"design": design, "size": size, "layers": n_layers, "prompt": prompt, "batch": batch,
            "l2": "weights of a step, and the inputs of a timed kernel, exceed L2",
            "models": whole_model(design, size, prompt, steps, batch, n_layers)}
    for d in line["models"].values():
        if "decode_bytes_per_step" in d:
            d["decode_frac_of_hbm_peak"] = round(d["decode_bytes_per_step"] / (d["decode_us_per_step"] * 1e-6) / (gbs * 1e9), 3)
    if kernels:
        def table(fn, *args):
            t = Table(gbs, tflops)
            fn(t, *args)
            return t.rows
        with torch.no_grad():
            if design == "femirax":
                line["decode_kernels"] = table(femirax_kernels, size, batch, 1, prompt)
                line["prompt_kernels"] = table(femirax_kernels, size, prompt, prompt, prompt)
                line["closest_model_kernels"] = table(decode_kernels, size, prompt, batch) + table(prompt_kernels, size, prompt)
            else:
                line["decode_kernels"] = table(decode_kernels, size, prompt, batch)
                line["prompt_kernels"] = table(prompt_kernels, size, prompt)
                line["closest_model_kernels"] = table(like_kernels, size, prompt, prompt)
    line["kernel_self_check"] = dense.debug_error()
    return line
