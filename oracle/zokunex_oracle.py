"""Plain, slow implementation of the Zokunex decoder in torch on the CPU: what the tests compare the product path with.

One function per mechanism, token by token where the mechanism is a recurrence, with nothing shared with
``glorcq_b200``.  ``W`` maps tensor names to tensors; everything is evaluated in the dtype of ``W`` (float32 or
float64 in the tests).
"""

from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    mu = x.mean(-1, keepdim=True)
    d = x - mu
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def log_gate_input(h, w, b, cap):
    """i = cap tanh((w h + b) / cap)"""
    return cap * torch.tanh((h @ w.T + b) / cap)


def log_gate_forget(h, w, b, cap):
    return torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w.T + b) / cap))


def mlstm_state(cfg, dtype=torch.float64):
    H, D, V = cfg["heads"], cfg["dim"], cfg["vdim"]
    return {"S": torch.zeros(H, D, V, dtype=dtype), "n": torch.zeros(H, D, dtype=dtype), "m": torch.zeros(H, dtype=dtype)}


def mlstm_recurrence(q, k, v, i, f, state):
    """q, k (T, H, D), v (T, H, V), log gates i, f (T, H); ``state`` is advanced in place.  Returns (T, H, V)."""
    out = []
    S, n, m = state["S"], state["n"], state["m"]
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(num / den[:, None])
    state["S"], state["n"], state["m"] = S, n, m
    return torch.stack(out)


def mlstm_mixer(h, W, p, cfg, eps, state):
    T = h.shape[0]
    H, D, V = cfg["heads"], cfg["dim"], cfg["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, D)
    v = (h @ W[p + "v"].T).view(T, H, V)
    i = log_gate_input(h, W[p + "i"], W[p + "i.b"], cfg["gate_cap"])
    f = log_gate_forget(h, W[p + "f"], W[p + "f.b"], cfg["gate_cap"])
    o = rms(mlstm_recurrence(q, k, v, i, f, state), eps).reshape(T, H * V)
    return (o * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def rotate(x, positions, base, dims):
    """x (T, ..., n): pairs (i, i + dims/2) of the first ``dims`` entries turned by position * base^(-2i/dims)."""
    half = dims // 2
    a = positions.to(torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = torch.cos(a).to(x.dtype).view(shape), torch.sin(a).to(x.dtype).view(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def latent_state(cfg, dtype=torch.float64):
    return {"c": torch.zeros(0, cfg["kv_rank"], dtype=dtype), "r": torch.zeros(0, cfg["rot_dim"], dtype=dtype)}


def causal_attention(q, k, v, scale, start):
    """q (T, H, D) at positions start.., k (S, H, D), v (S, H, V) -> (T, H, V)"""
    T, S = q.shape[0], k.shape[0]
    s = torch.einsum("thd,shd->hts", q, k) * scale
    seen = torch.arange(S)[None, :] <= start + torch.arange(T)[:, None]
    s = s.masked_fill(~seen[None], -math.inf)
    return torch.einsum("hts,shv->thv", torch.softmax(s, -1), v)


def latent_attention_mixer(h, W, p, cfg, eps, state):
    T, start = h.shape[0], state["c"].shape[0]
    H, D, R, V, K = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    base, dims = cfg["rot"]["base"], cfg["rot"]["dims"]
    pos = start + torch.arange(T)
    q = (h @ W[p + "q"].T).view(T, H, D + R)
    q = torch.cat([q[..., :D], rotate(q[..., D:], pos, base, dims)], -1)
    ckr = h @ W[p + "dkv"].T
    c = rms(ckr[:, :K], eps) * W[p + "dkv.norm"]
    state["c"] = torch.cat([state["c"], c])
    state["r"] = torch.cat([state["r"], rotate(ckr[:, K:], pos, base, dims)])
    S = state["c"].shape[0]
    k = (state["c"] @ W[p + "uk"].T).view(S, H, D)
    k = torch.cat([k, state["r"][:, None, :].expand(S, H, R)], -1)
    v = (state["c"] @ W[p + "uv"].T).view(S, H, V)
    o = causal_attention(q, k, v, cfg["scale"], start)
    o = o * torch.sigmoid(h @ W[p + "g"].T)[..., None]
    return o.reshape(T, H * V) @ W[p + "o"].T


def dense_ff(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def route(h, W, p, top):
    """(chosen experts (T, top), their weights): largest softmax score plus correction, weighted by the bare score."""
    s = torch.softmax(h @ W[p + "router"].T, -1)
    sel = torch.topk(s + W[p + "correction"], top, -1).indices
    return sel, torch.gather(s, 1, sel)


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def moe_ff(h, W, p, router):
    n = router["experts"]
    sel, wt = route(h, W, p, router["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(sel[t].tolist(), wt[t]):
            y[t] += w * (gelu_erf(h[t] @ W[p + f"e{e}.up"].T) @ W[p + f"e{e}.down"].T if e < n else h[t])
    return y


def new_state(cfg, dtype=torch.float64):
    return [(mlstm_state if L["type"] == "mlstm" else latent_state)(L["mixer"], dtype) for L in cfg["layers"]]


def forward(cfg, W, tokens, state, trace=None):
    """Logits (T, vocab) of the tokens that follow ``state`` (advanced in place); ``trace`` collects the residual
    stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for l, L in enumerate(cfg["layers"]):
        mixer = {"mlstm": mlstm_mixer, "latent_attention": latent_attention_mixer}[L["type"]]
        x = x + layer_norm(mixer(x, W, f"l{l}.mix.", L["mixer"], eps, state[l]), W[f"l{l}.norm1"], eps)
        if L.get("mlp"):
            p = f"l{l}.mlp."
            y = dense_ff(x, W, p) if L["mlp"]["kind"] == "dense" else moe_ff(x, W, p, L["mlp"]["router"])
            x = x + layer_norm(y, W[f"l{l}.norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]
