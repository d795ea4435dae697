"""Plain, slow implementation of the Femirax decoder in torch on the CPU: what the tests compare the product path with.

One function per mechanism, token by token where the mechanism is a recurrence, with nothing shared with
``glorcq_b200``.  ``W`` maps tensor names to tensors; everything is evaluated in the dtype of ``W`` (float32 or
float64 in the tests).
"""

from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def _angles(positions, base, dims, like, x_dim):
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = positions.to(torch.float64)[:, None] * f
    shape = (len(positions),) + (1,) * (x_dim - 2) + (dims // 2,)
    return torch.cos(a).to(like.dtype).view(shape), torch.sin(a).to(like.dtype).view(shape)


def rotate_halves(x, positions, base, dims):
    """x (T, ..., n): entries i and i + dims/2 of the first ``dims`` turned by position * base^(-2i/dims)."""
    c, s = _angles(positions, base, dims, x, x.dim())
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def rotate_pairs(x, positions, base, dims):
    """The same with entries 2i and 2i + 1 as the pair."""
    c, s = _angles(positions, base, dims, x, x.dim())
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def decayed_recurrence(q, k, v, alpha, S):
    """S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t.  q, k (T, H, D), v (T, H, V), alpha broadcastable to (T, H, D);
    S (H, D, V) is advanced in place.  Returns (T, H, V)."""
    T, H, D = q.shape
    alpha = alpha.expand(T, H, D)
    out = []
    for t in range(T):
        S.copy_(alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :])
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def retention_mixer(h, W, p, m, eps, state):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = state["n"] + torch.arange(T)
    rot = m["rot"]
    q = rotate_halves((h @ W[p + "q"].T).view(T, H, D), pos, rot["base"], rot["dims"])
    k = rotate_halves((h @ W[p + "k"].T).view(T, H, D), pos, rot["base"], rot["dims"]) * D ** -0.5
    v = (h @ W[p + "v"].T).view(T, H, V)
    decay = torch.tensor(m["decay"], dtype=h.dtype)[None, :, None]
    o = rms(decayed_recurrence(q, k, v, decay, state["S"]), eps).reshape(T, H * V)
    state["n"] += T
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def shared_value_attention(h, W, p, m, eps, state):
    """Grouped-query attention whose values are the projected keys; queries and keys are turned, then divided by their
    root mean square."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    start = state["k"].shape[0]
    pos = start + torch.arange(T)
    rot = m["rot"]
    raw = (h @ W[p + "k"].T).view(T, G, D)
    q = rms(rotate_pairs((h @ W[p + "q"].T).view(T, H, D), pos, rot["base"], rot["dims"]), eps)
    k = rms(rotate_pairs(raw, pos, rot["base"], rot["dims"]), eps)
    state["k"], state["v"] = torch.cat([state["k"], k]), torch.cat([state["v"], raw])
    o = causal_attention(q, state["k"], state["v"], m["scale"], start)
    return o.reshape(T, -1) @ W[p + "o"].T


def causal_attention(q, k, v, scale, start):
    """q (T, H, D) at positions start.., k (S, G, D), v (S, G, V) -> (T, H, V); head h reads head h // (H/G)."""
    T, H = q.shape[:2]
    S, G = k.shape[:2]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("thd,shd->hts", q, k) * scale
    seen = torch.arange(S)[None, :] <= start + torch.arange(T)[:, None]
    return torch.einsum("hts,shv->thv", torch.softmax(s.masked_fill(~seen[None], -math.inf), -1), v)


def gated_linear_attention(h, W, p, m, eps, state):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, D)
    v = (h @ W[p + "v"].T).view(T, H, V)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = torch.exp(torch.nn.functional.logsigmoid(z) / m["tau"]).view(T, H, D)
    o = rms(decayed_recurrence(q, k, v, alpha, state["S"]), eps) * W[p + "norm"]
    return (o.reshape(T, H * V) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel_mixer(h, W, p, m, eps, state):
    left = shared_value_attention(h, W, p + "left.", m["left"], eps, state["left"])
    right = gated_linear_attention(h, W, p + "right.", m["right"], eps, state["right"])
    return 0.5 * (rms(left, eps) * W[p + "left.out"] + rms(right, eps) * W[p + "right.out"])


def gated_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def token_side(x, e, W, p, eps):
    """x plus what the token's own row e of the layer gives"""
    y = (gelu_tanh(x @ W[p + "gate"].T) * e) @ W[p + "proj"].T
    return x + rms(y, eps) * W[p + "norm"]


def recurrent_state(m, dtype):
    return {"S": torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=dtype), "n": 0}


def key_state(m, dtype):
    return {"k": torch.zeros(0, m["kv_heads"], m["dim"], dtype=dtype), "v": torch.zeros(0, m["kv_heads"], m["dim"], dtype=dtype)}


def new_state(cfg, dtype=torch.float64):
    out = []
    for L in cfg["layers"]:
        m = L["mixer"]
        out.append(recurrent_state(m, dtype) if L["type"] == "retention" else
                   {"left": key_state(m["left"], dtype), "right": recurrent_state(m["right"], dtype)})
    return out


def forward(cfg, W, tokens, state, trace=None):
    """Logits (T, vocab) of the tokens that follow ``state`` (advanced in place); ``trace`` collects the residual
    stream after every layer."""
    eps, n = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][ids]
    for l, L in enumerate(cfg["layers"]):
        mixer = {"retention": retention_mixer, "parallel": parallel_mixer}[L["type"]]
        x = x + mixer(rms(x, eps) * W[f"l{l}.norm1"], W, f"l{l}.mix.", L["mixer"], eps, state[l])
        if L.get("mlp"):
            x = x + gated_ff(rms(x, eps) * W[f"l{l}.norm2"], W, f"l{l}.mlp.")
        x = token_side(x, W["side.embed"][ids][:, l * n:(l + 1) * n], W, f"l{l}.side.", eps)
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T
