"""Plain, slow restatement of the Vegodra design in PyTorch on the CPU: one function per mechanism.

Test infrastructure only; it shares no code with the product path (``pegainfer_b200/vegodra.py`` and the CUDA kernels
behind it).  Weights are a dict ``name -> tensor`` with the checkpoint's tensor names, configuration is the parsed
``config.json`` dict.  Everything runs in one floating type (fp32, or fp64 where ``dtype`` says so); attention is the dense
[queries x keys] form with an explicit visibility matrix, the latent attention expands keys and values per head (the product
path never does), the recurrence runs token by token.

Vegodra: x_0 = ln(embed[token]);  every layer reads one layer norm (weight and bias) of the residual and adds the sum of both sublayers,

    h = ln(x);   x <- x + (mixer(h) + ff(h)),

logits = head ln(x).  Mixers: latent attention (queries through a normed latent, interleaved rotary part shared by the heads, an
element-wise logistic output gate), chunked grouped-query attention (half-split rotation, then unit-RMS queries and keys, a learned sink
per head, one logistic output gate per head, optionally another layer's keys and values) and gated linear attention (a decay per key
channel, read-out normed per head and gated by SiLU).  Feed-forward: W_down(gelu_tanh(W_gate h) * (W_up h)), or none.
"""
from __future__ import annotations

import math

import torch

F32 = torch.float32


# ---------------------------------------------------------------- norms and activations
def rms(x, eps: float):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps: float):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * weight.to(x.dtype) + bias.to(x.dtype)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------- positions
def angles(pos, dims: int, base: float):
    """[T, dims / 2] in fp64"""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    return pos.to(torch.float64)[:, None] * f[None, :]


def turn(u, v, a):
    c, s = torch.cos(a).to(u.dtype), torch.sin(a).to(u.dtype)
    return u * c - v * s, v * c + u * s


def rotate_halves(x, pos, rot):
    """x [T, heads, d]: entry i turns with entry i + dims / 2; entries from ``dims`` on pass unchanged"""
    dims = int(rot["dims"])
    h = dims // 2
    u, v = turn(x[..., :h], x[..., h:dims], angles(pos, dims, rot["base"])[:, None, :])
    return torch.cat([u, v, x[..., dims:]], -1)


def rotate_neighbours(x, pos, rot):
    """x [T, heads, d]: entry 2i turns with entry 2i + 1; entries from ``dims`` on pass unchanged"""
    dims = int(rot["dims"])
    u, v = turn(x[..., 0:dims:2], x[..., 1:dims:2], angles(pos, dims, rot["base"])[:, None, :])
    return torch.cat([torch.stack([u, v], -1).flatten(-2), x[..., dims:]], -1)


# ---------------------------------------------------------------- attention
def visible(pos_q, pos_k, chunk: int):
    """[queries, keys] bool: keys up to the query's position, with a chunk size only those of the query's own chunk"""
    ok = pos_q[:, None] >= pos_k[None, :]
    if chunk:
        ok &= torch.div(pos_q, chunk, rounding_mode="floor")[:, None] == torch.div(pos_k, chunk, rounding_mode="floor")[None, :]
    return ok


def softmax_over(s, ok, sink=None):
    """weights of the visible keys; a sink is one more score that carries no value"""
    s = torch.where(ok, s, torch.full_like(s, -float("inf")))
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, sink.to(s.dtype).expand(s.shape[0], 1)], -1), -1)[:, :-1]


def keys_and_values(h, w, pre, mx, pos, eps):
    """what a layer with projections of its own caches: rotated unit-RMS keys [T, G, dim] and values [T, G, vdim]"""
    G, D, Dv = mx["kv_heads"], mx["dim"], mx["vdim"]
    k = (h @ w[pre + "k"].to(h.dtype).T).reshape(-1, G, D)
    return rms(rotate_halves(k, pos, mx["rot"]), eps), (h @ w[pre + "v"].to(h.dtype).T).reshape(-1, G, Dv)


def chunked_attention(q, k, v, mx, pos, sink):
    """q [T, H, dim], k [S, G, dim], v [S, G, vdim] of one sequence with positions 0 .. S - 1; queries at ``pos``"""
    H, G = q.shape[1], k.shape[1]
    ok = visible(pos, torch.arange(k.shape[0]), int((mx.get("mask") or {}).get("size", 0)))
    return torch.stack([softmax_over((q[:, i] @ k[:, i // (H // G)].T) * mx["scale"], ok, sink[i]) @ v[:, i // (H // G)] for i in range(H)], 1)


def attention_mixer(h, w, pre, mx, pos, eps, kv=None):
    """-> (result, (k, v)); ``kv``: another layer's keys and values in place of the layer's own"""
    H, D = mx["heads"], mx["dim"]
    q = rms(rotate_halves((h @ w[pre + "q"].to(h.dtype).T).reshape(-1, H, D), pos, mx["rot"]), eps)
    k, v = kv if kv is not None else keys_and_values(h, w, pre, mx, pos, eps)
    o = chunked_attention(q, k, v, mx, pos, w[pre + "sink"])
    o = o * torch.sigmoid(h @ w[pre + "g"].to(h.dtype).T)[:, :, None]
    return o.flatten(1) @ w[pre + "o"].to(h.dtype).T, (k, v)


def latent_mixer(h, w, pre, mx, pos, eps):
    H, D, R, Dv, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    W = lambda n: w[pre + n].to(h.dtype)  # noqa: E731
    cq = rms(h @ W("dq").T, eps) * W("dq.norm")
    q = (cq @ W("uq").T).reshape(-1, H, D + R)
    d = h @ W("dkv").T
    c = rms(d[:, :rank], eps) * W("dkv.norm")
    kr = rotate_neighbours(d[:, None, rank:], pos, mx["rot"])[:, 0]
    qr = rotate_neighbours(q[..., D:], pos, mx["rot"])
    k, v = (c @ W("uk").T).reshape(-1, H, D), (c @ W("uv").T).reshape(-1, H, Dv)
    ok = visible(pos, pos, 0)
    o = torch.stack([softmax_over((q[:, i, :D] @ k[:, i].T + qr[:, i] @ kr.T) * mx["scale"], ok) @ v[:, i] for i in range(H)], 1)
    return (o.flatten(1) * torch.sigmoid(h @ W("g").T)) @ W("o").T


# ---------------------------------------------------------------- gated linear attention
def channel_decay(z, tau: float):
    return torch.sigmoid(z) ** (1.0 / tau)


def decayed_memory(q, k, v, alpha, S=None):
    """q, k, alpha [T, H, dim], v [T, H, vdim] -> (o [T, H, vdim], S [H, dim, vdim])"""
    T, H, D = k.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=v.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gla_mixer(h, w, pre, mx, eps, S=None):
    """-> (result, state)"""
    H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
    W = lambda n: w[pre + n].to(h.dtype)  # noqa: E731
    q, k, v = (h @ W("q").T).reshape(-1, H, D) * D ** -0.5, (h @ W("k").T).reshape(-1, H, D), (h @ W("v").T).reshape(-1, H, Dv)
    alpha = channel_decay(h @ W("a1").T @ W("a2").T + W("a2.b"), mx["tau"]).reshape(-1, H, D)
    o, S = decayed_memory(q, k, v, alpha, S)
    o = (rms(o, eps) * W("norm")).flatten(1) * silu(h @ W("g").T)
    return o @ W("o").T, S


# ---------------------------------------------------------------- the model
def feed_forward(h, w, pre):
    W = lambda n: w[pre + n].to(h.dtype)  # noqa: E731
    return (gelu_tanh(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def forward(cfg, w, tokens, trail=None, dtype=F32):
    """logits [T, vocab] of one whole sequence; ``trail`` collects the residual after every layer"""
    w = {n: t.to(dtype) for n, t in w.items()}
    eps = float(cfg["norm"]["eps"])
    norm = lambda x, n: layer_norm(x, w[n], w[n + ".b"], eps)  # noqa: E731
    pos = torch.arange(len(tokens))
    x = norm(w["embed"][torch.as_tensor(tokens)], "embed.norm")
    cached = {}
    for i, l in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", l["mixer"]
        h = norm(x, p + "norm1")
        if l["type"] == "latent_attention":
            y = latent_mixer(h, w, p + "mix.", mx, pos, eps)
        elif l["type"] == "attention":
            src = mx.get("kv_from")
            y, cached[i] = attention_mixer(h, w, p + "mix.", mx, pos, eps, None if src is None else cached[src])
        elif l["type"] == "gla":
            y, _ = gla_mixer(h, w, p + "mix.", mx, eps)
        else:
            raise ValueError(l["type"])
        if l.get("mlp"):
            y = y + feed_forward(h, w, p + "mlp.")
        x = x + y
        if trail is not None:
            trail.append(x)
    return norm(x, "final.norm") @ w["head"].T
