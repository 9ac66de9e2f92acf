"""Plain, slow restatement of the Rilonex design in PyTorch on the CPU: one function per mechanism.

Test infrastructure only; it shares no code with the product path (``pegainfer_b200/rilonex.py`` and the CUDA kernels
behind it).  Weights are a dict ``name -> tensor`` with the checkpoint's tensor names, configuration is the parsed
``config.json`` dict.  Everything runs in one floating type (fp32, or fp64 where ``dtype`` says so); attention is the dense
[queries x keys] form with an explicit visibility matrix, every recurrence runs token by token.

Rilonex: a pre-norm decoder whose residual is a set of ``streams`` parallel rows.  A sublayer reads one weighted sum of
the streams; its result is added to every stream with a weight of its own while the streams are mixed by a small matrix.
Mixers:

* ``rglru`` -- a gated linear recurrent unit, one scalar state per channel, behind a short causal convolution; its gates are
  block-diagonal projections of the convolved input; the read-out is multiplied by a GELU branch.
* ``channel_delta`` -- the gated delta rule with a decay per head AND key channel (a low-rank projection), unit queries and keys
  behind short convolutions, read-out RMS-normed per head and gated by a low-rank logistic projection.
* ``parallel`` -- attention beside a gated delta rule with one decay per head, summed with two constants.  The attention mixes its
  heads' scores with a matrix, weighs a visible key by the logistic of (score + a bias per head) without normalising over keys,
  and multiplies every head's output by one logistic gate.

Feed-forward: W_down(relu(W_gate h) * (W_up h)), or none.
"""
from __future__ import annotations

import math

import torch

F32 = torch.float32
UNIT_EPS = 1e-6       # inside the root of the unit-vector normalisation of q and k
DECAY_RATE = 8.0      # rglru: log a = -DECAY_RATE * r * softplus(lam)


def rms(x, eps: float):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------- positions and attention
def rotate_halves(x, pos, rot):
    """x [T, heads, d]: entry i pairs with entry i + dims / 2 (i < dims / 2); entries from ``dims`` on pass unchanged."""
    if not rot or int(rot["dims"]) == 0:
        return x
    dims, half = int(rot["dims"]), int(rot["dims"]) // 2
    f = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    a = pos.to(torch.float64)[:, None] * f[None, :]
    cos, sin = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def mixed_scores(q, k, scale: float, talk):
    """[H, T, S]: scaled scores of every head (head h reads key head h // (H / G)), then score_h <- sum_g talk[h, g] score_g."""
    H, G = q.shape[1], k.shape[1]
    s = torch.stack([(q[:, h] @ k[:, h // (H // G)].T) * scale for h in range(H)])
    return torch.einsum("hg,gts->hts", talk, s)


def logistic_weights(scores, head_bias, pos_q, pos_k):
    """weight of a visible key: logistic(score + bias of the head); an invisible key weighs nothing; rows are not normalised."""
    ok = pos_q[:, None] >= pos_k[None, :]
    return torch.where(ok[None], torch.sigmoid(scores + head_bias[:, None, None]), torch.zeros_like(scores))


def talking_attention(h, w, pre, mx, pos):
    """Left branch of ``parallel`` for one sequence (all keys of the sequence are among the rows)."""
    H, G, D, Dv = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    W = lambda n: w[pre + n].to(h.dtype)  # noqa: E731
    q = rotate_halves((h @ W("q").T).reshape(-1, H, D), pos, mx.get("rot"))
    k = rotate_halves((h @ W("k").T).reshape(-1, G, D), pos, mx.get("rot"))
    v = (h @ W("v").T).reshape(-1, G, Dv)
    p = logistic_weights(mixed_scores(q, k, float(mx["scale"]), W("talk")), W("pb"), pos, pos)
    o = torch.stack([p[hd] @ v[:, hd // (H // G)] for hd in range(H)], 1)          # [T, H, Dv]
    o = o * torch.sigmoid(h @ W("g").T)[:, :, None]
    return o.reshape(-1, H * Dv) @ W("o").T


# ---------------------------------------------------------------- recurrences
def causal_conv(x, weight, bias=None, tail=None):
    """x [T, C]; weight [C, taps] whose LAST column multiplies the current token; zeros (or ``tail`` [taps - 1, C]) before the start.
    Returns (output, the new tail)."""
    taps = weight.shape[1]
    xp = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype) if tail is None else tail, x], 0)
    out = torch.zeros_like(x) if bias is None else bias.expand(x.shape[0], -1).clone()
    for j in range(taps):
        out = out + xp[j:j + x.shape[0]] * weight[:, j]
    return out, xp[x.shape[0]:]


def linear_unit(u, r, i, lam, S=None):
    """u, r, i [T, C]: S <- a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); returns (S after every token, last S)."""
    S = torch.zeros(u.shape[1], dtype=u.dtype) if S is None else S
    out = []
    for t in range(u.shape[0]):
        a = torch.exp(-DECAY_RATE * r[t] * softplus(lam))
        S = a * S + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        out.append(S)
    return torch.stack(out), S


def block_diagonal(x, m, b):
    """x [T, nb * n], m [nb, n (out), n (in)], b [nb, n]"""
    nb, n = m.shape[0], m.shape[1]
    return (torch.einsum("boi,tbi->tbo", m, x.reshape(-1, nb, n)) + b).reshape(-1, nb * n)


def gated_linear_mixer(h, w, pre, mx, state=None):
    """The ``rglru`` mixer; ``state`` = (S [width], conv tail) or None.  Returns (output, new state)."""
    W = lambda n: w[pre + n].to(h.dtype)  # noqa: E731
    S, tail = (None, None) if state is None else state
    y = gelu_tanh(h @ W("y").T + W("y.b"))
    u, tail = causal_conv(h @ W("x").T + W("x.b"), W("conv"), W("conv.b"), tail)
    r = torch.sigmoid(block_diagonal(u, W("ra"), W("ra.b")))
    i = torch.sigmoid(block_diagonal(u, W("ri"), W("ri.b")))
    out, S = linear_unit(u, r, i, W("lam"), S)
    return (out * y) @ W("o").T, (S, tail)


def delta_rule(q, k, v, g, beta, S=None):
    """q, k [T, H, D] (unit vectors, q scaled), v [T, H, Dv], g [T, H, D] decay of every key channel, beta [T, H].
    S [H, D, Dv]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, D = k.shape
    S = torch.zeros(H, D, v.shape[2], dtype=k.dtype) if S is None else S
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_mixer(h, w, pre, mx, eps, per_channel: bool, state=None):
    """The ``channel_delta`` mixer (per_channel) or the right branch of ``parallel`` (one decay per head).  ``state`` = (S, tails of
    q, k, v) or None.  Returns (output, new state)."""
    H, G, D, Dv = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    W = lambda n: w[pre + n].to(h.dtype)  # noqa: E731
    S, tails = (None, (None, None, None)) if state is None else state
    T = h.shape[0]
    seq, new_tails = [], []
    for n, t in zip("qkv", tails):
        c, nt = causal_conv(h @ W(n).T, W(n + ".conv"), None, t)
        seq.append(silu(c))
        new_tails.append(nt)
    rep = torch.arange(H) // (H // G)
    q = (unit(seq[0].reshape(T, G, D)) * D ** -0.5)[:, rep]
    k = unit(seq[1].reshape(T, G, D))[:, rep]
    v = seq[2].reshape(T, H, Dv)
    beta = torch.sigmoid(h @ W("b").T)
    rate = torch.exp(W("A_log"))
    if per_channel:
        z = ((h @ W("a1").T) @ W("a2").T + W("dt_bias")).reshape(T, H, D)
        g = torch.exp(-rate[:, None] * softplus(z))
        gate = torch.sigmoid((h @ W("g1").T) @ W("g2").T)
    else:
        g = torch.exp(-rate * softplus(h @ W("a").T + W("dt_bias")))[:, :, None].expand(T, H, D)
        gate = silu(h @ W("g").T)
    o, S = delta_rule(q, k, v, g, beta, S)
    o = (rms(o, eps) * W("norm")).reshape(T, H * Dv) * gate
    return o @ W("o").T, (S, tuple(new_tails))


def parallel_mixer(h, w, pre, mx, pos, eps):
    left = talking_attention(h, w, pre + "left.", mx["left"], pos)
    right, _ = delta_mixer(h, w, pre + "right.", mx["right"], eps, False)
    return float(mx["left_scale"]) * left + float(mx["right_scale"]) * right


def gated_relu(h, w, pre):
    return (torch.relu(h @ w[pre + "gate"].to(h.dtype).T) * (h @ w[pre + "up"].to(h.dtype).T)) @ w[pre + "down"].to(h.dtype).T


# ---------------------------------------------------------------- the residual streams
def read_streams(x, w_in):
    """x [streams, T, width] -> sum_s w_in[s] x_s"""
    return torch.einsum("s,stw->tw", w_in, x)


def write_streams(x, y, mix, out):
    """x_t <- sum_s mix[s, t] x_s + out[t] y  (mix is indexed [from, to]; all streams from the old ones)"""
    return torch.einsum("st,snw->tnw", mix, x) + out[:, None, None] * y[None]


def forward(cfg, w, tokens, trail=None, dtype=F32):
    """Logits [T, vocab] of one sequence from position 0; ``trail`` (a list) receives the sum of the streams after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    toks = torch.as_tensor(tokens)
    pos = torch.arange(len(toks))
    n = int(cfg["streams"])
    x = w["embed"][toks].expand(n, -1, -1).clone()
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(read_streams(x, w[p + "hc1.in"]), eps) * w[p + "norm1"]
        kind, mx = layer["type"], layer["mixer"]
        if kind == "rglru":
            y, _ = gated_linear_mixer(h, w, p + "mix.", mx)
        elif kind == "channel_delta":
            y, _ = delta_mixer(h, w, p + "mix.", mx, eps, True)
        elif kind == "parallel":
            y = parallel_mixer(h, w, p + "mix.", mx, pos, eps)
        else:
            raise ValueError(kind)
        x = write_streams(x, y, w[p + "hc1.mix"], w[p + "hc1.out"])
        if layer.get("mlp"):
            h = rms(read_streams(x, w[p + "hc2.in"]), eps) * w[p + "norm2"]
            x = write_streams(x, gated_relu(h, w, p + "mlp."), w[p + "hc2.mix"], w[p + "hc2.out"])
        if trail is not None:
            trail.append(x.sum(0))
    return (rms(x.sum(0), eps) * w["final.norm"]) @ w["head"].T
