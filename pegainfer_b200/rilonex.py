"""The Rilonex design on the layer-list host (``pegainfer_b200/layered.py``, csrc/host/layered_host.cpp).

Rilonex is a pre-norm decoder whose ``config.json`` lists its layers one by one.  Its residual is ``streams`` parallel rows x_s (fp32,
all equal to the embedding at the start).  A sublayer with the weights ``in``, ``out``, ``mix`` (``l<i>.hc1.*`` for the mixer,
``l<i>.hc2.*`` for the feed-forward) computes

    u = sum_s in[s] x_s;   y = sublayer(rms(u) * w);   x_t <- sum_s mix[s, t] x_s + out[t] y        rms(v) = v / sqrt(mean(v^2) + eps)

and the sum of the streams passes the last norm and the output head.  A configuration without ``streams`` has the ordinary residual
``x <- x + y`` and no such tensors.  Three mixers:

* ``rglru`` -- a real-gated linear recurrent unit: ``u = conv(W_x h + b_x)`` (short causal convolution per channel, with bias, no
  activation); per channel ``S <- a S + sqrt(1 - a^2) i u`` with ``log a = -8 r softplus(lam)`` and logistic gates r, i that are
  block-diagonal projections of u; the result is ``W_o (S * gelu_tanh(W_y h + b_y))``.
* ``channel_delta`` -- the gated delta rule with one decay per head and key channel, ``g = exp(-exp(A_log) softplus(W_a2 W_a1 h +
  dt_bias))``: ``S <- g S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q``; q, k, v pass short convolutions and SiLU, q and k are unit
  vectors; o is RMS-normed per head and multiplied by ``logistic(W_g2 W_g1 h)``.
* ``parallel`` -- two branches on the same input, ``left_scale * left + right_scale * right``.  Left: grouped-query attention whose
  scaled scores are mixed over the heads by a matrix (``talk``); the weight of a visible key is ``logistic(score + pb[h])``, not
  normalised over keys; each head's output is multiplied by one logistic gate; the first ``rot.dims`` entries of q and k rotate in
  half-split pairs.  Paged K/V cache.  Right: the gated delta rule with one decay per head and a ``silu(W_g h)`` read-out gate.

Recurrent states (fp32) and the convolutions' last inputs live in a per-request state slot.  The feed-forward, where a layer has one, is
``W_down (relu(W_gate h) * (W_up h))``.  The ranks of the low-rank projections are given by their tensors' shapes.

All sizes and constants come from the configuration or from the tensors; nothing here depends on one particular checkpoint.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace

import torch

from .layered import LayerCfg, LayeredModel, ModelCfg

MIXER_KINDS = {"channel_delta": 2, "rglru": 5, "parallel": 6}
DECAY_RATE = 8.0  # of the linear recurrent unit, fixed by the design


@dataclass(frozen=True)
class MixedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0        # 0: nothing rotates
    rot_base: float = 1.0

    @staticmethod
    def parse(d: dict) -> "MixedAttentionConfig":
        rot = d.get("rot") or {}
        return MixedAttentionConfig(int(d["heads"]), int(d.get("kv_heads") or d["heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]),
                                    int(rot.get("dims", 0)), float(rot.get("base", 1.0)))

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot_dims:
            d["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return d


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int = 0      # channel_delta: from the shape of 'a1'
    gate_rank: int = 0       # channel_delta: from the shape of 'g1'

    @staticmethod
    def parse(d: dict) -> "DeltaConfig":
        return DeltaConfig(int(d["heads"]), int(d.get("kv_heads") or d["heads"]), int(d["dim"]), int(d["vdim"]), int(d["conv"]))

    def to_dict(self) -> dict:
        return {k: getattr(self, k) for k in ("heads", "kv_heads", "dim", "vdim", "conv")}


@dataclass(frozen=True)
class LinearUnitConfig:
    width: int
    blocks: int
    conv: int

    @staticmethod
    def parse(d: dict) -> "LinearUnitConfig":
        return LinearUnitConfig(int(d["width"]), int(d["blocks"]), int(d["conv"]))

    def to_dict(self) -> dict:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass(frozen=True)
class RilonexLayerConfig:
    kind: str                                # "rglru" | "channel_delta" | "parallel"
    attention: MixedAttentionConfig | None   # left branch of "parallel"
    delta: DeltaConfig | None                # right branch of "parallel", or the mixer itself
    unit: LinearUnitConfig | None            # "rglru"
    left_scale: float
    right_scale: float
    ff: int                                  # 0: no feed-forward

    @staticmethod
    def parse(l: dict) -> "RilonexLayerConfig":
        kind, m, f = l["type"], l["mixer"], l.get("mlp")
        if kind not in MIXER_KINDS:
            raise ValueError(f"unknown mixer type {kind!r}")
        if f and f.get("kind") != "dense":
            raise ValueError(f"unknown feed-forward kind {f.get('kind')!r}")
        par = kind == "parallel"
        return RilonexLayerConfig(kind, MixedAttentionConfig.parse(m["left"]) if par else None,
                                  DeltaConfig.parse(m["right"]) if par else DeltaConfig.parse(m) if kind == "channel_delta" else None,
                                  LinearUnitConfig.parse(m) if kind == "rglru" else None, float(m["left_scale"]) if par else 1.0,
                                  float(m["right_scale"]) if par else 1.0, int(f["ff"]) if f else 0)

    def to_dict(self) -> dict:
        if self.kind == "parallel":
            m = {"left": self.attention.to_dict(), "right": self.delta.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}
        else:
            m = (self.unit or self.delta).to_dict()
        return {"type": self.kind, "mixer": m, "mlp": {"kind": "dense", "ff": self.ff} if self.ff else None}


@dataclass(frozen=True)
class RilonexConfig:
    vocab: int
    width: int
    eps: float
    streams: int             # 0: the ordinary residual
    layers: tuple = field(default_factory=tuple)
    name: str = "custom"

    @staticmethod
    def from_dict(raw: dict, name: str = "custom") -> "RilonexConfig":
        return RilonexConfig(int(raw["vocab"]), int(raw["width"]), float(raw["norm"]["eps"]), int(raw.get("streams") or 0),
                             tuple(RilonexLayerConfig.parse(l) for l in raw["layers"]), name)

    def to_dict(self) -> dict:
        """The ``config.json`` form (round-trips through ``from_dict``, apart from the ranks that the tensors give)."""
        d = {"architecture": "Rilonex", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": [l.to_dict() for l in self.layers]}
        if self.streams:
            d["streams"] = self.streams
        return d


def with_ranks(c: RilonexConfig, shapes: dict) -> RilonexConfig:
    """The ranks of every channel_delta layer's low-rank projections, read off the shapes of 'a1' and 'g1'."""
    layers = list(c.layers)
    for i, l in enumerate(layers):
        if l.kind != "channel_delta":
            continue
        ranks = [shapes.get(f"l{i}.mix.{n}") for n in ("a1", "g1")]
        if all(r is None for r in ranks) and l.delta.decay_rank and l.delta.gate_rank:
            continue
        if any(r is None for r in ranks):
            raise KeyError(f"l{i}: channel_delta needs the tensors mix.a1 and mix.g1")
        layers[i] = replace(l, delta=replace(l.delta, decay_rank=int(ranks[0][0]), gate_rank=int(ranks[1][0])))
    return replace(c, layers=tuple(layers))


def weight_shapes(c: RilonexConfig) -> dict:
    """Checkpoint tensor name -> shape (linear weights are [out, in])."""
    W, S = c.width, c.streams
    s = {"embed": (c.vocab, W)}
    for i, l in enumerate(c.layers):
        p = f"l{i}."
        s[p + "norm1"] = (W,)
        if l.ff:
            s[p + "norm2"] = (W,)
        m = p + "mix."
        if l.kind == "rglru":
            C, nb = l.unit.width, l.unit.blocks
            for n in ("y", "x"):
                s[m + n], s[m + n + ".b"] = (C, W), (C,)
            s[m + "conv"], s[m + "conv.b"] = (C, l.unit.conv), (C,)
            for n in ("ra", "ri"):
                s[m + n], s[m + n + ".b"] = (nb, C // nb, C // nb), (nb, C // nb)
            s[m + "lam"], s[m + "o"] = (C,), (W, C)
        else:
            if l.kind == "parallel":
                a, left = l.attention, m + "left."
                s[left + "q"], s[left + "k"], s[left + "v"] = (a.heads * a.dim, W), (a.kv_heads * a.dim, W), (a.kv_heads * a.vdim, W)
                s[left + "talk"], s[left + "pb"], s[left + "g"], s[left + "o"] = (a.heads, a.heads), (a.heads,), (a.heads, W), (W, a.heads * a.vdim)
                m += "right."
            d = l.delta
            for n, rows in (("q", d.kv_heads * d.dim), ("k", d.kv_heads * d.dim), ("v", d.heads * d.vdim)):
                s[m + n], s[m + n + ".conv"] = (rows, W), (rows, d.conv)
            s[m + "b"], s[m + "A_log"], s[m + "norm"] = (d.heads, W), (d.heads,), (d.vdim,)
            if l.kind == "parallel":
                s[m + "a"], s[m + "dt_bias"], s[m + "g"] = (d.heads, W), (d.heads,), (d.heads * d.vdim, W)
            else:
                s[m + "a1"], s[m + "a2"], s[m + "dt_bias"] = (d.decay_rank, W), (d.heads * d.dim, d.decay_rank), (d.heads * d.dim,)
                s[m + "g1"], s[m + "g2"] = (d.gate_rank, W), (d.heads * d.vdim, d.gate_rank)
            s[m + "o"] = (W, d.heads * d.vdim)
        if l.ff:
            s[p + "mlp.gate"], s[p + "mlp.up"], s[p + "mlp.down"] = (l.ff, W), (l.ff, W), (W, l.ff)
        for q in (1, 2) if S and l.ff else (1,) if S else ():
            s[f"{p}hc{q}.in"], s[f"{p}hc{q}.out"], s[f"{p}hc{q}.mix"] = (S,), (S,), (S, S)
    s["final.norm"] = (W,)
    s["head"] = (c.vocab, W)
    return s


def iter_random_weights(c: RilonexConfig, seed: int = 0, device: str = "cpu"):
    """Random-init checkpoint (bf16): projections N(0, 1/fan_in) so activations stay O(1); norm weights near one; stream weights near an
    even split; recurrence parameters of order one; attention biases far enough below zero that a sum over many keys stays O(1)."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)

    def rn(shape, std=1.0):
        return std * torch.randn(shape, generator=g, device=device)

    for name, shape in weight_shapes(c).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.1 * rn(shape)
        elif leaf == "conv":
            t = rn(shape, 0.5)
        elif leaf == "A_log":
            t = rn(shape, 0.5) - 1.0
        elif leaf in ("dt_bias", "lam"):
            t = rn(shape, 0.5) - 1.0
        elif leaf == "pb":
            t = rn(shape, 0.3) - 6.0
        elif leaf == "talk":
            t = torch.eye(shape[0], device=device) + rn(shape, 0.2)
        elif leaf == "in":
            t = 1.0 / shape[0] + rn(shape, 0.1)
        elif leaf == "out":
            t = 1.0 + rn(shape, 0.1)
        elif leaf == "mix":
            t = torch.eye(shape[0], device=device) + rn(shape, 0.05)
        elif leaf == "b" and len(shape) < 3 and name.count(".") > 2 and name.split(".")[-2] in ("y", "x", "conv", "ra", "ri"):
            t = rn(shape, 0.2)
        elif name == "embed":
            t = rn(shape)
        else:
            t = rn(shape) / shape[-1] ** 0.5
        yield name, t.to(torch.bfloat16)


# ---------------------------------------------------------------- the model class
def _layer_struct(l: RilonexLayerConfig) -> LayerCfg:
    a, d, u = l.attention, l.delta, l.unit
    s = LayerCfg(mixer_kind=MIXER_KINDS[l.kind], kv_from=-1, weights_of=-1, mlp_kind=int(l.ff > 0), ff=l.ff, mlp_act=1, rot_base=1.0, scale=1.0,
                 left_scale=l.left_scale, right_scale=l.right_scale)
    if a:
        s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.rot_dims, s.rot_base = a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.rot_dims, a.rot_base
    if d:
        s.d_heads, s.d_kv_heads, s.d_dim, s.d_vdim, s.conv, s.decay_rank, s.gate_rank = d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.decay_rank, d.gate_rank
    if u:
        s.lru_width, s.lru_blocks, s.conv, s.lru_rate = u.width, u.blocks, u.conv, DECAY_RATE
    return s


def _model_struct(cfg: RilonexConfig, mc: ModelCfg) -> ModelCfg:
    mc.block_kind, mc.streams = 4, cfg.streams
    return mc


class RilonexModel(LayeredModel):
    architecture = "Rilonex"
    config_class = RilonexConfig
    weight_shapes = staticmethod(weight_shapes)
    complete_config = staticmethod(with_ranks)
    layer_struct = staticmethod(_layer_struct)
    model_struct = staticmethod(_model_struct)
