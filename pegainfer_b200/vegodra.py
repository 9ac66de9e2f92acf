"""The Vegodra design on the layer-list host (``pegainfer_b200/layered.py``, csrc/host/layered_host.cpp).

Vegodra is a decoder whose ``config.json`` lists its layers one by one.  The embedding passes a layer norm (weight and bias); every
layer reads ONE layer norm of the fp32 residual and adds the sum of its two sublayers:

    h = ln(x);   x <- x + (mixer(h) + ff(h))          ln(v) = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w + b

Three mixers:

* ``latent_attention`` -- queries and keys / values pass RMS-normed latents (``dq``, ``dkv``); a score is the sum of an unrotated product
  per head and a rotated one (pairs (2i, 2i + 1)) whose key part all heads share; softmax over all earlier positions; the heads' outputs are
  multiplied entry by entry with ``logistic(W_g h)``.  The paged cache holds the kv latent and the rotated key part only.
* ``attention`` -- grouped-query attention whose queries and keys rotate (pairs (i, i + dims / 2)) and are then divided by their root
  mean square per head; chunk-local causal mask (``mask.size``), a learned sink per head, one logistic output gate per head.  A layer with
  ``kv_from`` has no keys and values of its own and reads that layer's cache.
* ``gla`` -- gated linear attention: per head ``S <- diag(a) S + k v^T``, ``o = S^T q / sqrt(dim)`` with ``a = logistic(W_a2 W_a1 h +
  b)^(1 / tau)`` per key channel; the read-out is RMS-normed per head and multiplied by ``silu(W_g h)``.  fp32 state slot per request.

The feed-forward, where a layer has one, is ``W_down (gelu_tanh(W_gate h) * (W_up h))``.  The rank of the decay's projection is given by its
tensors' shapes.  All sizes and constants come from the configuration or from the tensors; nothing here depends on one particular checkpoint.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace

import torch

from .layered import LayerCfg, LayeredModel, ModelCfg

MIXER_KINDS = {"latent_attention": 0, "attention": 1, "gla": 7}
GATE_ELEMENTS, GATE_HEADS = 1, 2   # LayerCfg.out_gate
UNIT_RMS = 3                       # LayerCfg.qk_norm
GELU_GATE = 2                      # LayerCfg.mlp_act


@dataclass(frozen=True)
class VegodraMixerConfig:
    kind: str                # "latent_attention" | "attention" | "gla"
    heads: int
    dim: int                 # query / key size per head (latent_attention: its unrotated part)
    vdim: int
    kv_heads: int = 0        # attention
    scale: float = 1.0       # attention, latent_attention
    chunk: int = 0           # attention: mask.size (0: every earlier position)
    kv_from: int = -1        # attention: the layer whose keys and values this one reads (-1: its own)
    rot_dims: int = 0
    rot_base: float = 1.0
    q_rank: int = 0          # latent_attention
    kv_rank: int = 0         # latent_attention
    rot_dim: int = 0         # latent_attention: size of the rotated part
    tau: float = 1.0         # gla
    decay_rank: int = 0      # gla: from the shape of 'a1'

    @staticmethod
    def parse(kind: str, d: dict) -> "VegodraMixerConfig":
        if kind not in MIXER_KINDS:
            raise ValueError(f"unknown mixer type {kind!r}")
        rot = d.get("rot") or {}
        common = dict(kind=kind, heads=int(d["heads"]), dim=int(d["dim"]), vdim=int(d["vdim"]), rot_dims=int(rot.get("dims", 0)),
                      rot_base=float(rot.get("base", 1.0)))
        if kind == "latent_attention":
            return VegodraMixerConfig(**common, scale=float(d["scale"]), q_rank=int(d["q_rank"]), kv_rank=int(d["kv_rank"]), rot_dim=int(d["rot_dim"]))
        if kind == "attention":
            src = d.get("kv_from")
            return VegodraMixerConfig(**common, scale=float(d["scale"]), kv_heads=int(d.get("kv_heads") or d["heads"]),
                                      chunk=int((d.get("mask") or {}).get("size", 0)), kv_from=-1 if src is None else int(src))
        return VegodraMixerConfig(**common, tau=float(d["tau"]))

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}
        if self.rot_dims:
            d["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        if self.kind == "latent_attention":
            d.update(scale=self.scale, q_rank=self.q_rank, kv_rank=self.kv_rank, rot_dim=self.rot_dim)
        elif self.kind == "attention":
            d.update(scale=self.scale, kv_heads=self.kv_heads)
            if self.chunk:
                d["mask"] = {"size": self.chunk}
            if self.kv_from >= 0:
                d["kv_from"] = self.kv_from
        else:
            d["tau"] = self.tau
        return d


@dataclass(frozen=True)
class VegodraLayerConfig:
    mixer: VegodraMixerConfig
    ff: int                  # 0: no feed-forward

    @staticmethod
    def parse(l: dict) -> "VegodraLayerConfig":
        f = l.get("mlp")
        if f and f.get("kind") != "dense":
            raise ValueError(f"unknown feed-forward kind {f.get('kind')!r}")
        return VegodraLayerConfig(VegodraMixerConfig.parse(l["type"], l["mixer"]), int(f["ff"]) if f else 0)


@dataclass(frozen=True)
class VegodraConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple = field(default_factory=tuple)
    name: str = "custom"

    @staticmethod
    def from_dict(raw: dict, name: str = "custom") -> "VegodraConfig":
        return VegodraConfig(int(raw["vocab"]), int(raw["width"]), float(raw["norm"]["eps"]), tuple(VegodraLayerConfig.parse(l) for l in raw["layers"]), name)

    def to_dict(self) -> dict:
        """The ``config.json`` form (round-trips through ``from_dict``, apart from the rank that the tensors give)."""
        return {"architecture": "Vegodra", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "layers": [{"type": l.mixer.kind, "mixer": l.mixer.to_dict(), "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]}


def with_ranks(c: VegodraConfig, shapes: dict) -> VegodraConfig:
    """The rank of every gla layer's decay projection, read off the shape of 'a1'."""
    layers = list(c.layers)
    for i, l in enumerate(layers):
        if l.mixer.kind != "gla":
            continue
        a1 = shapes.get(f"l{i}.mix.a1")
        if a1 is None:
            if l.mixer.decay_rank:
                continue
            raise KeyError(f"l{i}: gla needs the tensor mix.a1")
        layers[i] = replace(l, mixer=replace(l.mixer, decay_rank=int(a1[0])))
    return replace(c, layers=tuple(layers))


def weight_shapes(c: VegodraConfig) -> dict:
    """Checkpoint tensor name -> shape (linear weights are [out, in])."""
    W = c.width
    s = {"embed": (c.vocab, W)}

    def norm(name):
        s[name], s[name + ".b"] = (W,), (W,)

    norm("embed.norm")
    for i, l in enumerate(c.layers):
        m, p = l.mixer, f"l{i}.mix."
        H, D, Dv = m.heads, m.dim, m.vdim
        norm(f"l{i}.norm1")
        if m.kind == "latent_attention":
            s[p + "dq"], s[p + "dq.norm"], s[p + "uq"] = (m.q_rank, W), (m.q_rank,), (H * (D + m.rot_dim), m.q_rank)
            s[p + "dkv"], s[p + "dkv.norm"] = (m.kv_rank + m.rot_dim, W), (m.kv_rank,)
            s[p + "uk"], s[p + "uv"], s[p + "g"] = (H * D, m.kv_rank), (H * Dv, m.kv_rank), (H * Dv, W)
        elif m.kind == "attention":
            s[p + "q"], s[p + "sink"], s[p + "g"] = (H * D, W), (H,), (H, W)
            if m.kv_from < 0:
                s[p + "k"], s[p + "v"] = (m.kv_heads * D, W), (m.kv_heads * Dv, W)
        else:
            s[p + "q"], s[p + "k"], s[p + "v"], s[p + "g"], s[p + "norm"] = (H * D, W), (H * D, W), (H * Dv, W), (H * Dv, W), (Dv,)
            s[p + "a1"], s[p + "a2"], s[p + "a2.b"] = (m.decay_rank, W), (H * D, m.decay_rank), (H * D,)
        s[p + "o"] = (W, H * Dv)
        if l.ff:
            s[f"l{i}.mlp.gate"], s[f"l{i}.mlp.up"], s[f"l{i}.mlp.down"] = (l.ff, W), (l.ff, W), (W, l.ff)
    norm("final.norm")
    s["head"] = (c.vocab, W)
    return s


def iter_random_weights(c: VegodraConfig, seed: int = 0, device: str = "cpu"):
    """Random-init checkpoint (bf16): projections N(0, 1/fan_in) so activations stay O(1); norm weights near one, their biases small; sinks and decay
    biases of order one."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)

    def rn(shape, std=1.0):
        return std * torch.randn(shape, generator=g, device=device)

    for name, shape in weight_shapes(c).items():
        if name.endswith((".norm", ".norm1")):
            t = 1.0 + rn(shape, 0.1)
        elif name.endswith(("norm.b", "norm1.b")):
            t = rn(shape, 0.1)
        elif name.endswith("a2.b"):
            t = 1.0 + rn(shape)
        elif len(shape) == 1 or name == "embed":
            t = rn(shape)
        else:
            t = rn(shape) / shape[1] ** 0.5
        yield name, t.to(torch.bfloat16)


# ---------------------------------------------------------------- the model class
def _layer_struct(l: VegodraLayerConfig) -> LayerCfg:
    m = l.mixer
    s = LayerCfg(mixer_kind=MIXER_KINDS[m.kind], heads=m.heads, dim=m.dim, vdim=m.vdim, kv_from=m.kv_from, weights_of=-1, scale=m.scale, rot_dims=m.rot_dims,
                 rot_base=m.rot_base, mlp_kind=int(l.ff > 0), ff=l.ff, mlp_act=GELU_GATE)
    if m.kind == "latent_attention":
        s.q_rank, s.kv_rank, s.rot_dim, s.rot_interleaved, s.sink_kind, s.out_gate = m.q_rank, m.kv_rank, m.rot_dim, 1, 1, GATE_ELEMENTS
    elif m.kind == "attention":
        s.kv_heads, s.chunk, s.rot_interleaved, s.sink_kind, s.out_gate, s.qk_norm = m.kv_heads, m.chunk, 0, 0, GATE_HEADS, UNIT_RMS
    else:
        s.tau, s.decay_rank = m.tau, m.decay_rank
    return s


def _model_struct(cfg: VegodraConfig, mc: ModelCfg) -> ModelCfg:
    mc.block_kind = 5
    return mc


class VegodraModel(LayeredModel):
    architecture = "Vegodra"
    config_class = VegodraConfig
    weight_shapes = staticmethod(weight_shapes)
    complete_config = staticmethod(with_ranks)
    layer_struct = staticmethod(_layer_struct)
    model_struct = staticmethod(_model_struct)
