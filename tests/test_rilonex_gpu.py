"""Rilonex on the GPU against the plain oracle (oracle/rilonex_oracle.py): mechanisms alone through the C ABI or as one-layer
models, then the model through its own step / engine / generate entry points -- whole prompts, token-by-token decoding,
portions down to two tokens, unequal batches, reused pages and state slots, keys far back, at page and key-block borders and at the
query's own position, the first tokens, long decoding, greedy generation.

Configurations and weights are made here (small, random, seeded).  float32 runs are held to 2e-4 of the logits' spread
(against the oracle in fp64), bfloat16 runs to rounding noise.  Where random weights would blur a fault (one far key among
hundreds) the inputs are built so that a single score dominates.
"""
import math
import random

import pytest
import torch

from oracle import rilonex_oracle as O

pytestmark = pytest.mark.gpu

F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16


# ------------------------------------------------------------------ configurations (none is a real checkpoint's)
def lru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def chan(heads, kv_heads, dim, vdim, conv, ranks=(7, 10)):
    return {"type": "channel_delta", "mixer": delta(heads, kv_heads, dim, vdim, conv), "ranks": ranks}


def par(heads, kv_heads, dim, vdim, right, rot_dims=None, base=10000.0, scale=None, left_scale=0.7, right_scale=0.9):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    dims = dim if rot_dims is None else rot_dims
    if dims:
        left["rot"] = {"dims": dims, "base": base}
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def model_cfg(layers, vocab=211, width=88, eps=1e-5, streams=2):
    """layers: (mixer entry, hidden size of the feed-forward or 0).  The entry's 'ranks' (channel_delta: of the decay's and of the gate's
    projection) only shape the tensors; a checkpoint's config.json does not carry them."""
    return {"architecture": "Rilonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "layers": [dict(l, mlp={"kind": "dense", "ff": ff} if ff else None) for l, ff in layers]}


def cfg_general():
    """All sizes differ from each other; every mixer; a layer without feed-forward; in bf16 the first attention takes the tensor-core
    kernel (dim != vdim), the second the generic one."""
    return model_cfg([(par(6, 3, 32, 16, delta(4, 2, 24, 20, 3), rot_dims=20), 72), (lru(120, 5, 4), 56), (chan(6, 3, 12, 28, 2), 0),
                      (par(3, 1, 20, 36, delta(2, 2, 40, 12, 5), base=300.0, left_scale=1.3, right_scale=-0.4), 100)], streams=3)


def cfg_edges():
    """Values that often coincide or equal one are made to differ or to be one: one stream, one head, kv_heads == heads, one gate block and
    blocks of one channel, one-tap convolutions, ranks of one, no rotation, equal branch factors, widths that are no multiple of 4."""
    return model_cfg([(par(1, 1, 10, 7, delta(1, 1, 5, 9, 1), rot_dims=0, left_scale=1.0, right_scale=1.0), 0), (lru(27, 27, 1), 19), (lru(33, 1, 2), 0),
                      (chan(3, 3, 9, 11, 1, ranks=(1, 1)), 33), (par(5, 5, 6, 6, delta(3, 1, 7, 5, 2), rot_dims=6), 21)], vocab=97, width=50, eps=1e-6, streams=1)


def cfg_wide():
    """head sizes of the 128- and 256-wide register tiles, more heads than a tensor-core CTA sums, five streams, a long convolution"""
    return model_cfg([(par(18, 2, 16, 32, delta(2, 1, 96, 40, 12)), 64), (chan(2, 1, 160, 24, 3, ranks=(16, 24)), 40), (par(10, 5, 112, 128, delta(1, 1, 64, 64, 4)), 0),
                      (lru(64, 2, 11), 48)], vocab=128, width=64, streams=5)


def cfg_plain_residual():
    """no streams in the configuration: x <- x + y, no stream weights in the checkpoint"""
    c = model_cfg([(lru(48, 3, 3), 40), (par(4, 2, 16, 16, delta(2, 1, 16, 8, 4)), 32), (chan(2, 2, 8, 16, 4), 0)], vocab=80, width=40)
    del c["streams"]
    return c


CONFIGS = {"general": cfg_general, "edges": cfg_edges, "wide": cfg_wide, "plain_residual": cfg_plain_residual}


def config_of(cfg):
    """the product's configuration object with the ranks filled in (as the loader does from the tensors' shapes)"""
    from dataclasses import replace

    from pegainfer_b200.rilonex import RilonexConfig
    c = RilonexConfig.from_dict(cfg)
    return replace(c, layers=tuple(replace(l, delta=replace(l.delta, decay_rank=r["ranks"][0], gate_rank=r["ranks"][1])) if l.kind == "channel_delta" else l
                                   for l, r in zip(c.layers, cfg["layers"])))


def make_weights(cfg, seed, sharp=1.0):
    """bf16 checkpoint; `sharp` scales the attention's query projection so that single keys weigh far more than the rest"""
    from pegainfer_b200.rilonex import weight_shapes
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in weight_shapes(config_of(cfg)).items():
        leaf = name.rsplit(".", 1)[-1]
        rn = lambda s=1.0: s * torch.randn(shape, generator=g)  # noqa: E731
        if name.endswith("left.q"):
            t = sharp * rn() / math.sqrt(shape[1])
        elif leaf in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.2 * rn()
        elif leaf == "conv":
            t = rn(0.6)
        elif leaf in ("A_log", "lam", "dt_bias"):
            t = rn(0.8) - 1.5
        elif leaf == "pb":
            t = rn(0.5) - 4.0
        elif leaf == "talk":
            t = torch.eye(shape[0]) + rn(0.4 / math.sqrt(shape[0]))
        elif leaf == "in":
            t = 1.0 / shape[0] + rn(0.3)
        elif leaf == "out":
            t = 1.0 + rn(0.3)
        elif leaf == "mix":
            t = 0.7 * torch.eye(shape[0]) + rn(0.3)
        elif len(shape) == 1 or leaf == "b" and name.split(".")[-2] in ("ra", "ri"):
            t = rn(0.4)
        elif name == "embed":
            t = rn()
        else:
            t = rn() / math.sqrt(shape[-1])
        w[name] = t.to(BF16)
    return w


def build(cfg, w, dtype, max_tokens=1024, max_requests=4):
    from pegainfer_b200.rilonex import RilonexConfig, RilonexModel
    return RilonexModel(RilonexConfig.from_dict(cfg), w, dtype=dtype, max_tokens=max_tokens, max_requests=max_requests)


def row_errors(got, want):
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()


def close(got, want, dtype):
    """float32: every row within 2e-4 of the logits' spread.  bfloat16: rounding noise only (a wrong key, state or page shows in the
    float32 run of the same test)."""
    e = row_errors(got, want.to(F32))
    if dtype == F32:
        return e.max().item() < 2e-4
    return e.median().item() < 0.04 and e.quantile(0.9).item() < 0.10


SHARP = {F32: 4.0, BF16: 1.5}


def tokens_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def oracle_logits(cfg, w, toks, trail=None):
    if "streams" not in cfg:  # the ordinary residual is one stream with all its weights at one
        cfg, w = dict(cfg, streams=1), dict(w)
        for i, l in enumerate(cfg["layers"]):
            for q in (1, 2) if l["mlp"] else (1,):
                w[f"l{i}.hc{q}.in"] = w[f"l{i}.hc{q}.out"] = torch.ones(1)
                w[f"l{i}.hc{q}.mix"] = torch.ones(1, 1)
    return O.forward(cfg, w, toks, trail, dtype=F64)


# ------------------------------------------------------------------ kernels alone
@pytest.fixture(scope="module")
def lib():
    from pegainfer_b200 import ffi
    ffi.lib().cublas_init()
    return ffi.lib()


def dev(t, dtype):
    return t.to(dtype).cuda().contiguous()


def i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device="cuda")


class Hold:
    """ptr(t) returns t's device address and keeps t alive until the launches that read it are done."""

    def __init__(self):
        self.kept = []

    def __call__(self, t):
        self.kept.append(t)
        return t.data_ptr()


def rounded(t, dtype):
    return t.to(dtype).to(F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 7, 16])
@pytest.mark.parametrize("W", [50, 64, 4096, 13000])
def test_streams_are_read_and_written(lib, dtype, S, W):
    """embedding into all streams with the first read; write + next read; write without a next read; last norm over gathered rows; sum"""
    P = Hold()
    T, V, eps = 5, 9, 1e-5
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    f32 = int(dtype == F32)
    emb, y, wn = rounded(rnd(V, W), dtype), rounded(rnd(T, W), dtype), rounded(1 + 0.3 * rnd(W), dtype)
    win, wout, mix = rnd(S), rnd(S), rnd(S, S)
    ids = [3, 8, 0, 3, 7]
    x, h, h32 = torch.zeros(T, S, W, device="cuda"), torch.zeros(T, W, dtype=dtype, device="cuda"), torch.zeros(T, W, device="cuda")
    args = (x.data_ptr(), P(dev(wn, dtype)), h.data_ptr(), h32.data_ptr(), W, S, eps, T, f32, None)
    assert lib.pk_res32_streams_embed(P(dev(emb, dtype)), P(i32(ids)), P(win.cuda()), *args) == 0
    torch.cuda.synchronize()
    xs = emb[ids].expand(S, T, W)
    want = O.rms(O.read_streams(xs, win), eps) * wn
    assert torch.equal(x.cpu(), xs.transpose(0, 1))
    assert torch.allclose(h32.cpu(), want, atol=1e-5, rtol=1e-4)
    xs = rnd(S, T, W)
    x.copy_(xs.transpose(0, 1))
    assert lib.pk_res32_streams_step(P(dev(y, dtype)), P(mix.cuda()), P(wout.cuda()), P(win.cuda()), *args) == 0
    torch.cuda.synchronize()
    xs = O.write_streams(xs, y, mix, wout)
    want = O.rms(O.read_streams(xs, win), eps) * wn
    assert torch.allclose(x.cpu(), xs.transpose(0, 1), atol=2e-5)
    assert torch.allclose(h32.cpu(), want, atol=1e-4, rtol=1e-4)
    assert torch.allclose(h.float().cpu(), want, atol=1e-4 if dtype == F32 else 4e-2, rtol=1e-4 if dtype == F32 else 1e-2)
    assert lib.pk_res32_streams_step(P(dev(y, dtype)), P(mix.cuda()), P(wout.cuda()), None, x.data_ptr(), None, None, None, W, S, eps, T, f32, None) == 0
    rows = [4, 1, 1]
    out, total = torch.zeros(3, W, dtype=dtype, device="cuda"), torch.zeros(T, W, device="cuda")
    assert lib.pk_res32_streams_rows(x.data_ptr(), P(i32(rows)), P(dev(wn, dtype)), out.data_ptr(), None, W, S, eps, 3, f32, None) == 0
    assert lib.pk_res32_streams_rows(x.data_ptr(), None, None, None, total.data_ptr(), W, S, eps, T, f32, None) == 0
    torch.cuda.synchronize()
    xs = O.write_streams(xs, y, mix, wout)
    assert torch.allclose(total.cpu(), xs.sum(0), atol=1e-4 * S, rtol=1e-4)
    want = (O.rms(xs.sum(0), eps) * wn)[rows]
    assert torch.allclose(out.float().cpu(), want, atol=2e-4 if dtype == F32 else 4e-2, rtol=1e-3 if dtype == F32 else 1e-2)


def paged(req_lens, page_size, shuffle_seed=0):
    """A page table with pages handed out in a scrambled order: (pages flat, page_off per request, number of pages)."""
    need = [(n + page_size - 1) // page_size for n in req_lens]
    order = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(shuffle_seed)).tolist()
    pages, off, k = [], [], 0
    for n in need:
        off.append(len(pages))
        pages += order[k:k + n]
        k += n
    return pages, off, sum(need) + 3


def run_attention(lib, dtype, mx, qkv, talk, pb, gate, starts, lens, ps=16, max_kv=0, factor=1.0, shares=8):
    """rotation + cache append + attention for a step whose request r brings positions starts[r] .. lens[r] - 1 (earlier positions
    were appended by a first call); rows [q | k | v]; talk / pb / gate may be None; the workspace holds `shares` shares of the key axis.  Returns [T, H * vdim]."""
    P = Hold()
    H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    n_all = H * D + G * D + G * Dv
    pages, off, n_pages = paged(lens, ps, shuffle_seed=5)
    stride = ps * G * (D + Dv) + 24
    cache = torch.full((n_pages, stride), float("nan"), dtype=dtype, device="cuda")  # a slot that nothing wrote must not be read
    rot = mx.get("rot")
    dims = rot["dims"] if rot else 0
    freq = (float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)).to(F32).cuda() if rot else None
    f32 = int(dtype == F32)

    def step(rows_of):  # rows_of[r] = (first position, one past the last)
        x = torch.cat([qkv[r][a:b] for r, (a, b) in enumerate(rows_of)])
        p = [q for a, b in rows_of for q in range(a, b)]
        rq = [r for r, (a, b) in enumerate(rows_of) for _ in range(a, b)]
        T = len(p)
        if T == 0:
            return None
        ld = H * Dv + 6
        qo, out = torch.zeros(T, H * D, dtype=dtype, device="cuda"), torch.full((T, ld), 5.0, dtype=dtype, device="cuda")
        a = (P(i32(p)), P(i32(rq)), P(i32(off)), P(i32(pages)))
        gt = torch.cat([gate[r][s:e] for r, (s, e) in enumerate(rows_of)]) if gate is not None else None
        assert lib.pk_gqa_rope_append_ex(P(dev(x, dtype)), n_all, None, *a, qo.data_ptr(), cache.data_ptr(), stride, ps, H, G, D, Dv, dims, 0,
                                         freq.data_ptr() if rot else None, 1.0, 0.0, T, f32, None) == 0
        ws = torch.zeros(shares * T * H * Dv, device="cuda")
        assert lib.pk_gqa_mixed_attention(qo.data_ptr(), cache.data_ptr(), P(dev(talk, dtype)) if talk is not None else None,
                                          P(pb.cuda()) if pb is not None else None, P(gt.cuda()) if gt is not None else None, H + 2, *a, out.data_ptr(), ld,
                                          factor, stride, ps, T, H, G, D, Dv, float(mx["scale"]), max_kv, P(ws) if shares else None,
                                          4 * ws.numel(), f32, None) == 0
        torch.cuda.synchronize()
        assert (out[:, H * Dv:] == 5.0).all()  # nothing past the heads' columns is written
        return out[:, :H * Dv].float().cpu()

    step([(0, s) for s in starts])
    return step([(s, n) for s, n in zip(starts, lens)])


def oracle_attention(mx, qkv, talk, pb, gate, lo, hi, factor=1.0):
    """The oracle's mechanisms on a stacked projection output, in fp64."""
    H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    x = qkv[:hi].to(F64)
    pos = torch.arange(hi)
    q, k = O.rotate_halves(x[:, :H * D].reshape(-1, H, D), pos, mx.get("rot")), O.rotate_halves(x[:, H * D:(H + G) * D].reshape(-1, G, D), pos, mx.get("rot"))
    v = x[:, (H + G) * D:].reshape(-1, G, Dv)
    s = O.mixed_scores(q, k, mx["scale"], torch.eye(H, dtype=F64) if talk is None else talk.to(F64))
    p = O.logistic_weights(s, torch.zeros(H, dtype=F64) if pb is None else pb.to(F64), pos, pos)
    o = torch.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], 1)
    if gate is not None:
        o = o * torch.sigmoid(gate[:hi, :H].to(F64))[:, :, None]
    return (factor * o.reshape(hi, H * Dv))[lo:].to(F32)


# heads, kv heads, dim, vdim, rotated entries: bf16 with dim and vdim multiples of 16 up to 128 runs prompt portions on the tensor cores
ATTN_SHAPES = [(3, 1, 20, 12, 8), (6, 2, 32, 48, 32), (1, 1, 16, 16, 0), (4, 4, 64, 64, 16), (2, 1, 128, 128, 128), (9, 3, 32, 32, 32), (12, 4, 112, 16, 10),
               (16, 2, 80, 96, 80), (20, 4, 16, 32, 16), (34, 17, 16, 16, 4), (5, 5, 40, 72, 40), (8, 8, 96, 128, 96), (2, 2, 200, 256, 100)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,Dv,dims", ATTN_SHAPES)
def test_attention_ragged_batch(lib, dtype, H, G, D, Dv, dims):
    """three requests in one launch: a 70-token portion that starts at position 90, one decoded token at position 199, and the first 5
    tokens of a sequence; with and without a known longest context (the key axis is split); without mixing, biases and gate"""
    g = torch.Generator().manual_seed(3)
    mx = par(H, G, D, Dv, None, rot_dims=dims, scale=2.0 / math.sqrt(D))["mixer"]["left"]
    lens, starts = [160, 200, 5], [90, 199, 0]
    qkv = [rounded(torch.randn(n, (H + G) * D + G * Dv, generator=g), dtype) for n in lens]
    talk = rounded(torch.eye(H) + 0.5 * torch.randn(H, H, generator=g), dtype)
    pb, gate = torch.randn(H, generator=g) - 2.0, [torch.randn(n, H + 2, generator=g) for n in lens]
    for (t, b, gt, max_kv, shares) in ((talk, pb, gate, 0, 8), (talk, pb, gate, 200, 8), (talk, pb, gate, 200, 0), (None, None, None, 200, 2)):
        got = run_attention(lib, dtype, mx, qkv, t, b, gt, starts, lens, max_kv=max_kv, factor=-1.4, shares=shares)
        want = torch.cat([oracle_attention(mx, qkv[r], t, b, gt[r] if gt else None, starts[r], lens[r], -1.4) for r in range(3)])
        tol = 4e-5 if dtype == F32 else 2e-2
        assert (got - want).abs().max() < tol * max(1.0, want.abs().max().item()), max_kv


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D", [(4, 2, 32), (3, 3, 24)])
def test_decoded_tokens_of_unequal_contexts_in_one_launch(lib, dtype, H, G, D):
    """contexts of 1500, 130 and 2 positions: some shares of the key axis are empty for the short ones"""
    mx = par(H, G, D, D, None, rot_dims=8)["mixer"]["left"]
    g = torch.Generator().manual_seed(6)
    lens = [1500, 130, 2]
    starts = [n - 1 for n in lens]
    qkv = [rounded(torch.randn(n, (H + 2 * G) * D, generator=g), dtype) for n in lens]
    talk, pb = rounded(torch.eye(H) + 0.3 * torch.randn(H, H, generator=g), dtype), torch.full((H,), -5.0)
    want = torch.cat([oracle_attention(mx, qkv[r], talk, pb, None, starts[r], lens[r]) for r in range(3)])
    for max_kv, shares in ((0, 0), (1500, 100), (2048, 7)):
        got = run_attention(lib, dtype, mx, qkv, talk, pb, None, starts, lens, max_kv=max_kv, shares=shares)
        assert (got - want).abs().max() < (3e-5 if dtype == F32 else 1e-2) * max(1.0, want.abs().max().item()), max_kv


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("prompt", [False, True])
@pytest.mark.parametrize("H,D", [(2, 32), (2, 24), (10, 64)])
def test_single_keys_stand_out(lib, dtype, prompt, H, D):
    """One key is aimed at with a steep score and the bias makes every other key weigh nothing, so head 0's output must be that key's
    value and head 1, which asks nothing itself, gets the same through the mixing matrix.  Far keys, both sides of page borders (16) and
    of key-block borders (32), the first tokens, the query's own position; one past the query is hidden: nothing may come out.
    `prompt`: the query sits in a 40-token portion (bf16 with head sizes 32 / 64: tensor-core kernel), else it is a decoded token."""
    mx = par(H, 1, D, D, None, rot_dims=0, scale=40.0)["mixer"]["left"]
    n = 700
    g = torch.Generator().manual_seed(4)
    val = rounded(torch.randn(n, D, generator=g), dtype)
    key = torch.nn.functional.normalize(torch.randn(n, D, generator=g) - 0.0, dim=-1)
    pb = torch.full((H,), -20.0)
    talk = torch.eye(H)
    talk[1] = 0.0
    talk[1, 0] = 1.0  # head 1 listens to head 0
    cases = [(690, k) for k in (0, 1, 15, 16, 31, 32, 33, 63, 64, 300, 511, 512, 671, 672, 673, 687, 688, 689, 690, 691)] + \
            [(31, 31), (31, 0), (32, 31), (32, 32), (33, 32), (0, 0), (1, 0), (1, 1), (47, 48), (48, 48), (15, 16)]
    for q_at, kp in cases:
        qkv = torch.zeros(n, H * D + 2 * D)
        qkv[:, H * D:H * D + D], qkv[:, H * D + D:] = key, val
        qkv[:, H * D:H * D + D] *= 0.2
        qkv[kp, H * D:H * D + D] = key[kp]
        qkv[q_at, :D] = key[kp]
        qkv = rounded(qkv, dtype)
        hi = max(q_at, kp) + 1
        start = max(q_at - 39, 0) if prompt else q_at
        got = run_attention(lib, dtype, mx, [qkv], talk, pb, None, [start], [hi], max_kv=hi)[q_at - start]
        if kp <= q_at:
            assert torch.allclose(got[:D], val[kp], atol=2e-2, rtol=1e-2), (q_at, kp)
            assert torch.allclose(got[D:2 * D], val[kp], atol=2e-2, rtol=1e-2), (q_at, kp)
        else:
            assert got[:2 * D].abs().max() < 1e-2, (q_at, kp)
        if H > 2:
            assert got[2 * D:].abs().max() < 1e-3


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_weights_are_logistic_and_not_normalised(lib, dtype):
    """two cached positions, two heads: the arithmetic written out"""
    D = 16
    mx = par(2, 1, D, D, None, rot_dims=0, scale=0.3)["mixer"]["left"]
    g = torch.Generator().manual_seed(8)
    qkv = rounded(torch.randn(2, 4 * D, generator=g), dtype)
    talk, pb, gate = torch.tensor([[0.5, -1.0], [2.0, 0.25]]), torch.tensor([0.3, -0.6]), torch.tensor([[9.0, 9, 9, 9], [0.4, -1.1, 9, 9]])
    got = run_attention(lib, dtype, mx, [qkv], talk, pb, [gate], [1], [2], factor=0.8)[0]
    q, k, v = qkv[1, :2 * D].reshape(2, D), qkv[:, 2 * D:3 * D], qkv[:, 3 * D:]
    s = q @ k.T * 0.3                              # [head, key]
    z = torch.stack([0.5 * s[0] - 1.0 * s[1] + 0.3, 2.0 * s[0] + 0.25 * s[1] - 0.6])
    want = 0.8 * torch.sigmoid(gate[1, :2])[:, None] * (torch.sigmoid(z) @ v)
    assert torch.allclose(got, want.reshape(-1), atol=1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("taps", [1, 2, 4, 5, 12])
@pytest.mark.parametrize("act", [0, 1])
def test_convolution_carries_its_tail_through_portions(lib, dtype, taps, act):
    """two requests, fed in portions of 1, 2, 3, 19 and 7 tokens in turn (shorter and longer than the tail and than a group of
    tokens), slots swapped; with the input's bias (zeros, not the bias, stand before the start) and the output's, and without"""
    P = Hold()
    Cn, ld = 20, 27
    g = torch.Generator().manual_seed(5)
    xs = [rounded(torch.randn(n, Cn, generator=g), dtype) for n in (60, 45)]
    cw, cb, ib = [rounded(s * torch.randn(*sh, generator=g), dtype) for s, sh in ((0.7, (Cn, taps)), (0.5, (Cn,)), (0.8, (Cn,)))]
    for biased in (True, False):
        want = []
        for x in xs:
            y, _ = O.causal_conv(x + ib if biased else x, cw, cb if biased else None)
            want.append(O.silu(y) if act else y)
        slot_stride = 5 + max(taps - 1, 0) * Cn
        state = torch.zeros(3, slot_stride, device="cuda")
        slots, at, got = [2, 0], [0, 0], [[], []]
        sizes, k = [1, 2, 3, 19, 7], 0
        while any(at[r] < len(xs[r]) for r in range(2)):
            live = [r for r in range(2) if at[r] < len(xs[r])]
            ns = [min(sizes[(k + r) % 5], len(xs[r]) - at[r]) for r in live]
            rows = torch.zeros(sum(ns), ld)
            rows[:, 3:3 + Cn] = torch.cat([xs[r][at[r]:at[r] + n] for r, n in zip(live, ns)])
            row0 = [sum(ns[:e]) for e in range(len(ns))]
            out = torch.zeros(sum(ns), Cn, dtype=dtype, device="cuda")
            x_d = dev(rows, dtype)
            assert lib.pk_causal_conv(x_d.data_ptr() + 3 * x_d.element_size(), ld, P(dev(ib, dtype)) if biased else None, P(dev(cw, dtype)),
                                      P(dev(cb, dtype)) if biased else None, act, state.data_ptr() + 5 * 4, slot_stride, P(i32([slots[r] for r in live])),
                                      P(i32(row0)), P(i32(ns)), out.data_ptr(), Cn, Cn, taps, sum(ns), len(ns), int(dtype == F32), None) == 0
            torch.cuda.synchronize()
            o = out.float().cpu()
            for e, (r, n) in enumerate(zip(live, ns)):
                got[r].append(o[row0[e]:row0[e] + n])
                at[r] += n
            k += 1
        for r in range(2):
            assert torch.allclose(torch.cat(got[r]), want[r], atol=1e-5 if dtype == F32 else 3e-2, rtol=1e-5 if dtype == F32 else 1e-2), r
        assert state[1].abs().max().item() == 0.0 and state[:, :5].abs().max().item() == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Cn,blocks", [(24, 3), (50, 1), (40, 40), (17, 17)])
def test_linear_unit_in_portions_over_reused_slots(lib, dtype, Cn, blocks):
    """two sequences advance in portions of 1, 300, 9 and 40 tokens (token by token and scanned; more than one block of the scan)
    through slots 2 and 0; decays from nearly one to nearly zero"""
    P = Hold()
    g = torch.Generator().manual_seed(9)
    n, lens = Cn // blocks, [351, 700]
    us = [rounded(torch.randn(t, Cn, generator=g), dtype) for t in lens]
    ys = [rounded(2 * torch.randn(t, Cn, generator=g), dtype) for t in lens]
    zs = [2 * torch.randn(t, 2 * Cn + 3, generator=g) for t in lens]
    rb, ib, lam = torch.randn(Cn, generator=g), torch.randn(Cn, generator=g), 4 * torch.randn(Cn, generator=g) - 4.0
    yb = rounded(torch.randn(Cn, generator=g), dtype)
    want = []
    for u, y, z in zip(us, ys, zs):
        zz = z[:, :2 * Cn].to(F64).reshape(-1, blocks, 2, n)
        r, i = torch.sigmoid(zz[:, :, 0].reshape(-1, Cn) + rb), torch.sigmoid(zz[:, :, 1].reshape(-1, Cn) + ib)
        S, _ = O.linear_unit(u.to(F64), r, i, lam.to(F64))
        want.append((S * O.gelu_tanh(y.to(F64) + yb)).to(F32))
    state = torch.zeros(3, Cn + 3, device="cuda")
    slots, at, got = [2, 0], [0, 0], [[], []]
    sizes, k = [1, 300, 9, 40], 0
    while any(at[r] < lens[r] for r in range(2)):
        live = [r for r in range(2) if at[r] < lens[r]]
        ns = [min(sizes[(k + r) % 4], lens[r] - at[r]) for r in live]
        T = sum(ns)
        cut = lambda src: torch.cat([src[r][at[r]:at[r] + m] for r, m in zip(live, ns)])  # noqa: E731
        row0 = [sum(ns[:e]) for e in range(len(ns))]
        out = torch.full((T, Cn + 2), 3.0, dtype=dtype, device="cuda")
        assert lib.pk_lru_seq(P(dev(cut(us), dtype)), Cn, P(cut(zs).cuda()), 2 * Cn + 3, P(rb.cuda()), P(ib.cuda()), P(lam.cuda()), O.DECAY_RATE, blocks,
                              P(dev(cut(ys), dtype)), Cn, P(dev(yb, dtype)), state.data_ptr() + 4, Cn + 3, P(i32([slots[r] for r in live])), P(i32(row0)),
                              P(i32(ns)), out.data_ptr(), Cn + 2, Cn, T, len(ns), int(dtype == F32), None) == 0
        torch.cuda.synchronize()
        o = out.float().cpu()
        assert (o[:, Cn:] == 3.0).all()
        for e, (r, m) in enumerate(zip(live, ns)):
            got[r].append(o[row0[e]:row0[e] + m, :Cn])
            at[r] += m
        k += 1
    for r in range(2):
        assert torch.allclose(torch.cat(got[r]), want[r], atol=2e-5 if dtype == F32 else 2e-2, rtol=1e-4 if dtype == F32 else 1e-2), r
    assert state[1].abs().max().item() == 0.0 and state[:, 0].abs().max().item() == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,Dv", [(3, 1, 20, 24), (4, 4, 32, 48), (2, 1, 64, 100), (2, 2, 128, 16), (6, 3, 200, 8)])
@pytest.mark.parametrize("per_channel", [False, True])
def test_delta_rule_in_portions_over_reused_slots(lib, dtype, H, G, D, Dv, per_channel):
    """two sequences advance in portions of 1, 37 and 2 tokens through slots 2 and 0; one decay per head, or per head and key channel"""
    P = Hold()
    g = torch.Generator().manual_seed(10)
    lens = [45, 60]
    nq = G * D
    Cn = 2 * nq + H * Dv
    ld, ldz, ldc = Cn + 8, 2 * H + 3, H * D + 1
    xs = [rounded(torch.randn(n, Cn, generator=g), dtype) for n in lens]
    zs = [torch.randn(n, ldz, generator=g) for n in lens]
    zc = [2 * torch.randn(n, ldc, generator=g) for n in lens]
    a_log, dt = 0.7 * torch.randn(H, generator=g) - 1.0, 0.5 * torch.randn(H * D if per_channel else H, generator=g) - 1.0
    rep = torch.arange(H) // (H // G)
    want = []
    for x, z, c in zip(xs, zs, zc):
        x, z, c = x.to(F64), z.to(F64), c.to(F64)
        q, k = O.unit(x[:, :nq].reshape(-1, G, D))[:, rep] * D ** -0.5, O.unit(x[:, nq:2 * nq].reshape(-1, G, D))[:, rep]
        if per_channel:
            dec = torch.exp(-torch.exp(a_log.to(F64))[:, None] * O.softplus(c[:, :H * D] + dt).reshape(-1, H, D))
        else:
            dec = torch.exp(-torch.exp(a_log.to(F64)) * O.softplus(z[:, 1:1 + H] + dt))[:, :, None].expand(-1, H, D)
        o, _ = O.delta_rule(q, k, x[:, 2 * nq:].reshape(-1, H, Dv), dec, torch.sigmoid(z[:, 1 + H:1 + 2 * H]))
        want.append(o.reshape(-1, H * Dv).to(F32))
    stride = H * D * Dv + 11
    state = torch.zeros(3, stride, device="cuda")
    slots, at, got = [2, 0], [0, 0], [[], []]
    sizes, k = [1, 37, 2], 0
    while any(at[r] < lens[r] for r in range(2)):
        live = [r for r in range(2) if at[r] < lens[r]]
        ns = [min(sizes[(k + r) % 3], lens[r] - at[r]) for r in live]
        T = sum(ns)
        cut = lambda src: torch.cat([src[r][at[r]:at[r] + m] for r, m in zip(live, ns)])  # noqa: E731
        rows = torch.zeros(T, ld)
        rows[:, 8:] = cut(xs)
        row0 = [sum(ns[:e]) for e in range(len(ns))]
        out = torch.zeros(T, H * Dv, device="cuda")
        where = (state.data_ptr(), stride, P(i32([slots[r] for r in live])), P(i32(row0)), P(i32(ns)), out.data_ptr(), H, G, D, Dv, len(ns), int(dtype == F32), None)
        head = (P(dev(rows, dtype)), ld, 8, 8 + nq, 8 + 2 * nq, P(cut(zs).cuda()), ldz)
        if per_channel:
            c_d, ready = cut(zc).cuda(), k % 2  # every other step: the decays made by a launch of their own
            if ready:
                c_d = c_d[:, :H * D].contiguous()
                assert lib.pk_channel_decay(P(c_d), P(a_log.cuda()), P(dt.cuda()), T, H, D, None) == 0
            assert lib.pk_channel_delta_seq(*head, 1 + H, P(c_d), c_d.shape[1], ready, P(a_log.cuda()), P(dt.cuda()), *where) == 0
        else:
            assert lib.pk_gated_delta_seq(*head, 1, 1 + H, P(a_log.cuda()), P(dt.cuda()), *where) == 0
        torch.cuda.synchronize()
        o = out.cpu()
        for e, (r, m) in enumerate(zip(live, ns)):
            got[r].append(o[row0[e]:row0[e] + m])
            at[r] += m
        k += 1
    for r in range(2):
        assert torch.allclose(torch.cat(got[r]), want[r], atol=3e-5, rtol=1e-4), r
    assert state[1].abs().max().item() == 0.0  # the slot nobody owned is untouched


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows", [1, 8, 20, 70])
@pytest.mark.parametrize("batch,cols,K", [(3, 40, 24), (5, 14, 7), (1, 130, 64)])
def test_batched_product_with_fp32_results(lib, dtype, rows, batch, cols, K):
    """block-diagonal gates and low-rank second factors: strides of their own for both operands and the result"""
    P = Hold()
    g = torch.Generator().manual_seed(11)
    lda, ldc = batch * K + 8, batch * cols + 5
    A, B = rounded(torch.randn(rows, lda, generator=g), dtype), rounded(torch.randn(batch, cols, K, generator=g), dtype)
    C = torch.full((rows, ldc), 7.0, device="cuda")
    assert lib.pk_gemm_strided_f32out(P(dev(A, dtype)), P(dev(B, dtype)), C.data_ptr(), rows, cols, K, lda, K, ldc, batch, K, cols * K, cols, int(dtype == F32),
                                      None) == 0
    torch.cuda.synchronize()
    want = torch.einsum("rbk,bck->rbc", A[:, :batch * K].reshape(rows, batch, K), B).reshape(rows, -1)
    assert torch.allclose(C.cpu()[:, :batch * cols], want, atol=1e-4)  # bf16 operands, fp32 sums: no rounding of the result
    assert (C[:, batch * cols:] == 7.0).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,V", [(5, 14), (2, 300)])
@pytest.mark.parametrize("act", [0, 1])
def test_read_out_norm_with_stride_and_factor(lib, dtype, H, V, act):
    P = Hold()
    T, ld, ldo, off, eps = 6, H * V + 9, H * V + 4, 4, 1e-5
    g = torch.Generator().manual_seed(12)
    o, z, wn = 3 * torch.randn(T, H * V, generator=g), rounded(torch.randn(T, ld, generator=g), dtype), rounded(1 + 0.3 * torch.randn(V, generator=g), dtype)
    o[0] *= 1e-3  # of the order of sqrt(eps): the norm's eps shows
    out = torch.full((T, ldo), 2.0, dtype=dtype, device="cuda")
    assert lib.pk_head_norm_gate_ex(P(o.cuda()), None, P(dev(wn, dtype)), 0, P(dev(z, dtype)), ld, off, out.data_ptr(), ldo, -0.6, T, H, V, eps, act,
                                    int(dtype == F32), None) == 0
    torch.cuda.synchronize()
    zz = z[:, off:off + H * V]
    want = -0.6 * (O.rms(o.reshape(T, H, V), eps) * wn).reshape(T, -1) * (torch.sigmoid(zz) if act else O.silu(zz))
    assert torch.allclose(out[:, :H * V].float().cpu(), want, atol=1e-5 if dtype == F32 else 3e-2, rtol=1e-5 if dtype == F32 else 1e-2)
    assert (out[:, H * V:] == 2.0).all()


@pytest.mark.parametrize("T", [1, 4, 9, 300])
@pytest.mark.parametrize("W,ff", [(64, 96), (256, 520)])
def test_gate_and_up_projection_with_relu_in_the_epilogue(lib, T, W, ff):
    from pegainfer_b200.ffi import GemvArgs
    P = Hold()
    g = torch.Generator().manual_seed(13)
    x, wt = rounded(torch.randn(T, W, generator=g), BF16), rounded(torch.randn(2 * ff, W, generator=g) / math.sqrt(W), BF16)
    gate, up = rounded(x @ wt[:ff].T, BF16), rounded(x @ wt[ff:].T, BF16)
    want = torch.relu(gate) * up
    out = torch.zeros(T, ff, dtype=BF16, device="cuda")
    if T <= 4:
        a = GemvArgs()
        a.W, a.X, a.M, a.N, a.K, a.epi = P(dev(wt, BF16)), P(dev(x, BF16)), ff, T, W, 5
        a.Y[0], a.seg_rows[0] = out.data_ptr(), ff
        import ctypes as C
        assert lib.pk_b200_gemv_fused(C.byref(a), None) == 0
    else:
        rc = lib.pk_b200_gemm_gated(P(dev(wt, BF16)), P(dev(x, BF16)), out.data_ptr(), ff, T, W, 1, None)
        if rc == -2:
            pytest.skip("shape outside the fused kernel's range (the host then runs two launches)")
        assert rc == 0
    two = torch.zeros(T, ff, dtype=BF16, device="cuda")
    assert lib.pk_act(P(dev(torch.cat([gate, up], 1), BF16)), two.data_ptr(), ff, T, 2, 0, None) == 0
    torch.cuda.synchronize()
    assert torch.allclose(two.float().cpu(), want, atol=1e-6, rtol=1e-2)
    assert torch.allclose(out.float().cpu(), want, atol=2e-2, rtol=3e-2)
    assert (out[:, :] == 0).float().mean() > 0.3  # the gate's negative half is cut


# ------------------------------------------------------------------ one-layer models: each mixer and each branch alone
ONE = {"left": (par(4, 2, 16, 24, delta(3, 3, 8, 10, 3), right_scale=0.0), 0), "right": (par(4, 2, 16, 24, delta(4, 2, 20, 10, 3), left_scale=0.0), 0),
       "channel": (chan(4, 2, 20, 12, 4, ranks=(5, 3)), 0), "rglru": (lru(60, 3, 3), 0), "mlp": (par(1, 1, 8, 8, delta(1, 1, 8, 8, 2), left_scale=0.0, right_scale=0.0), 44)}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("which", sorted(ONE))
def test_each_mechanism_alone(dtype, which):
    """a portion, then decoded tokens; the output weight of the sublayer is large, so that its result dominates the streams"""
    cfg = model_cfg([ONE[which]], vocab=64, width=48, streams=2)
    w = make_weights(cfg, 14, SHARP[dtype])
    w["l0.hc1.out"], w["l0.hc1.mix"] = torch.tensor([3.0, -2.0]).to(BF16), (0.2 * w["l0.hc1.mix"].float()).to(BF16)
    toks = tokens_for(cfg, 90, 3)
    m = build(cfg, w, dtype)
    rid = m.alloc_request()
    got = torch.cat([m.step([(rid, toks[:50])], [list(range(50))])] + [m.step([(rid, [t])]) for t in toks[50:]])
    assert close(got, oracle_logits(cfg, w, toks), dtype)
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_read_outs_of_the_order_of_sqrt_eps(dtype):
    """value projections shrunk so that the norms' eps (layer and unit vectors) shows in the result"""
    cfg = model_cfg([(chan(2, 1, 12, 16, 2), 0), (par(2, 1, 8, 8, delta(2, 2, 12, 8, 2)), 0)], vocab=64, width=48, eps=1e-3)
    w = make_weights(cfg, 15)
    for n in ("l0.mix.v", "l1.mix.right.v", "l0.mix.q", "l1.mix.right.k"):
        w[n] = (w[n].float() * (2e-2 if n.endswith("v") else 1e-3)).to(BF16)
    toks = tokens_for(cfg, 60, 3)
    m = build(cfg, w, dtype)
    rid = m.alloc_request()
    got = torch.cat([m.step([(rid, toks[:40])], [list(range(40))])] + [m.step([(rid, [t])]) for t in toks[40:]])
    assert close(got, oracle_logits(cfg, w, toks), dtype)
    m.close()


# ------------------------------------------------------------------ the model through its own entry points
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_with_residual_after_every_layer(name, dtype):
    cfg = CONFIGS[name]()
    w = make_weights(cfg, 21, SHARP[dtype])
    toks = tokens_for(cfg, 150, 2)
    m = build(cfg, w, dtype)
    m.keep_trail(True)
    rid = m.alloc_request()
    got = m.step([(rid, toks)], [list(range(len(toks)))])
    trail = []
    want = oracle_logits(cfg, w, toks, trail)
    tr = m.trail(len(toks))
    assert len(trail) == len(cfg["layers"])
    for i, x in enumerate(trail):
        e = (tr[i] - x.to(F32)).abs().max() / x.abs().max()
        assert e < (1e-4 if dtype == F32 else 0.1), (i, e)
    assert close(got, want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_against_token_by_token_decoding(name, dtype):
    """the first tokens as one prompt, the rest one by one through the cache and the state slots; then the same sequence decoded
    from its very first token"""
    cfg = CONFIGS[name]()
    w = make_weights(cfg, 22, SHARP[dtype])
    toks = tokens_for(cfg, 130, 3)
    want = oracle_logits(cfg, w, toks)
    m = build(cfg, w, dtype)
    for first in (60, 1):
        rid = m.alloc_request()
        rows = [m.step([(rid, toks[:first])], [list(range(first))])]
        for t in range(first, len(toks)):
            rows.append(m.step([(rid, [toks[t]])]))
        assert close(torch.cat(rows), want, dtype), first
        m.drop_request(rid)
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["general", "wide"])
@pytest.mark.parametrize("sizes", [(2,), (3, 2, 16, 1, 37, 5), (64, 2, 2), (33, 1)])
def test_prompt_in_portions(name, dtype, sizes):
    """portions cut anywhere (inside pages, key blocks and the convolutions' tails), down to two tokens"""
    cfg = CONFIGS[name]()
    w = make_weights(cfg, 23, SHARP[dtype])
    toks = tokens_for(cfg, 140, 4)
    want = oracle_logits(cfg, w, toks)
    m = build(cfg, w, dtype)
    rid = m.alloc_request()
    rows, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - at)
        rows.append(m.step([(rid, toks[at:at + n])], [list(range(n))]))
        at, k = at + n, k + 1
    assert close(torch.cat(rows), want, dtype)
    m.close()


def random_cfg(seed):
    """layer order, every size and every constant drawn at random (seeded)"""
    r = random.Random(seed)

    def heads():
        h = r.choice([1, 2, 3, 4, 6, 8, 10, 12])
        return h, r.choice([d for d in range(1, h + 1) if h % d == 0])

    def some_delta():
        h, g = heads()
        return delta(h, g, r.choice([4, 8, 12, 20, 32, 40, 72, 130]), r.choice([4, 8, 16, 28, 48]), r.randint(1, 6))
    layers = []
    for _ in range(r.randint(2, 5)):
        kind = r.choice(["rglru", "channel_delta", "parallel"])
        if kind == "rglru":
            nb = r.choice([1, 2, 3, 5])
            l = lru(nb * r.choice([4, 8, 13, 16, 24]), nb, r.randint(1, 6))
        elif kind == "channel_delta":
            d = some_delta()
            l = {"type": kind, "mixer": d, "ranks": (r.randint(1, 30), r.choice([1, 6, 8, 16, 24]))}
        else:
            h, g = heads()
            dim = r.choice([8, 12, 16, 20, 32, 48, 64])
            l = par(h, g, dim, r.choice([8, 16, 28, 32, 64]), some_delta(), rot_dims=r.choice([0, 2, dim // 2 // 2 * 2, dim]),
                    base=r.choice([100.0, 10000.0, 500000.0]), scale=r.uniform(0.05, 0.4), left_scale=r.uniform(-1.5, 1.5), right_scale=r.uniform(-1.5, 1.5))
        layers.append((l, r.choice([0, 8, 20, 56, 88])))
    return model_cfg(layers, vocab=r.randint(40, 300), width=r.choice([24, 36, 41, 64, 100]), eps=r.choice([1e-5, 1e-6, 1e-3]), streams=r.choice([1, 2, 3, 4, 6]))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("seed", range(16))
def test_configurations_drawn_at_random(seed, dtype):
    """a prompt in portions of random sizes (some >= 32 tokens, so that the tensor-core kernels run where the sizes allow), then
    decoded tokens, against the oracle over the whole sequence"""
    cfg = random_cfg(100 + seed)
    w = make_weights(cfg, 200 + seed, SHARP[dtype])
    toks = tokens_for(cfg, 120, seed)
    want = oracle_logits(cfg, w, toks)
    m = build(cfg, w, dtype)
    rid = m.alloc_request()
    r = random.Random(seed)
    rows, at = [], 0
    while at < len(toks):
        n = 1 if at >= 100 else min(r.choice([1, 2, 5, 17, 33, 48]), 100 - at)
        rows.append(m.step([(rid, toks[at:at + n])], [list(range(n))]))
        at += n
    assert close(torch.cat(rows), want, dtype), cfg
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_batches_reuse_pages_and_slots(dtype):
    """Seven unequal requests through three request slots and a pool of 18 pages: portions of some beside single tokens of others in
    every step; finished requests hand their pages and state slot to the next one.  Every request must come out as when it runs alone."""
    from pegainfer_b200.engine import Engine
    cfg = cfg_general()
    w = make_weights(cfg, 24, SHARP[dtype])
    lens = [70, 9, 40, 101, 1, 33, 64]
    prompts = [tokens_for(cfg, n, 30 + i) for i, n in enumerate(lens)]
    want = [oracle_logits(cfg, w, p) for p in prompts]
    m = build(cfg, w, dtype, max_tokens=18 * 16, max_requests=3)
    eng = Engine(m)
    got = [[] for _ in prompts]
    at = [0] * len(prompts)
    waiting, live, step, seen_pages = list(range(len(prompts))), [], 0, set()
    portion = [5, 1, 17, 2, 1, 30, 3]
    pages_of = lambda i: (lens[i] + 15) // 16  # noqa: E731
    while waiting or live:
        while waiting and len(live) < 3 and sum(pages_of(i) for i in live) + pages_of(waiting[0]) <= 18:
            live.append(waiting.pop(0))
        entries = []
        for i in live:
            n = min(portion[(step + i) % len(portion)], lens[i] - at[i])
            entries.append((f"q{i}", prompts[i][at[i]:at[i] + n], list(range(n))))
        out = eng.step(entries, [])
        r = 0
        for (name, t, _), i in zip(entries, list(live)):
            got[i].append(out[r:r + len(t)])
            r += len(t)
            at[i] += len(t)
            seen_pages.update(m.request_pages(eng.slots[name]))
            if at[i] == lens[i]:
                eng.release(name)
                live.remove(i)
        step += 1
    assert sum((n + 15) // 16 for n in lens) > 18 >= len(seen_pages)  # pages were handed out again
    if dtype == BF16:  # a request of one token is one row: rounding is judged over all of them
        assert close(torch.cat([r for g in got for r in g]), torch.cat(want), dtype)
    for i in range(len(prompts)):
        assert dtype == BF16 or close(torch.cat(got[i]), want[i], dtype), i
    m.close()


def test_rejected_step_leaves_lengths_pages_and_state_untouched():
    cfg = cfg_general()
    w = make_weights(cfg, 25)
    toks = tokens_for(cfg, 60, 5)
    m = build(cfg, w, F32, max_tokens=64, max_requests=2)
    a, b = m.alloc_request(), m.alloc_request()
    m.step([(a, toks[:20])])
    free = m.available_pages()
    with pytest.raises(RuntimeError):
        m.step([(a, toks[20:25]), (b, toks[:60])])  # b does not fit: nothing of the step may stay
    assert m.seq_len(a) == 20 and m.seq_len(b) == 0 and m.available_pages() == free
    got = m.step([(a, toks[20:40])], [list(range(20))])
    assert close(got, oracle_logits(cfg, w, toks[:40])[20:], F32)
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_and_captured_steps(dtype):
    """a 300-token prompt and 260 decoded tokens (captured launch sequences from the second step of a kind on, across a graph bucket
    border at 512) against the same steps run eagerly and against the oracle"""
    cfg = model_cfg([(par(4, 2, 32, 32, delta(2, 1, 24, 16, 4), rot_dims=16), 32), (lru(48, 2, 4), 0), (chan(2, 2, 16, 16, 3), 40)], vocab=96, width=64, streams=4)
    w = make_weights(cfg, 26, SHARP[dtype])
    toks = tokens_for(cfg, 560, 6)
    outs = []
    for graph in (True, False):
        m = build(cfg, w, dtype, max_tokens=1024)
        m.use_graph(graph)
        rid = m.alloc_request()
        rows = [m.step([(rid, toks[:300])])]
        for t in range(300, 560):
            rows.append(m.step([(rid, [toks[t]])]))
        assert (m.graph_count() > 0) == graph
        outs.append(torch.cat(rows))
        m.close()
    assert torch.allclose(outs[0], outs[1], atol=1e-5 if dtype == F32 else 2e-2)
    want = oracle_logits(cfg, w, toks)[299:]
    assert close(outs[0], want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_batched_decode_steps_of_unequal_requests(dtype):
    """three prompts of unequal length admitted in one step, then 40 steps that carry one token of each (replayed as a captured
    launch sequence from the third step on); every request must come out as when it runs alone"""
    cfg = cfg_general()
    w = make_weights(cfg, 29, SHARP[dtype])
    lens = [23, 61, 4]
    seqs = [tokens_for(cfg, n + 40, 50 + i) for i, n in enumerate(lens)]
    want = [oracle_logits(cfg, w, q) for q in seqs]
    m = build(cfg, w, dtype)
    rids = [m.alloc_request() for _ in lens]
    got = [[] for _ in lens]
    out = m.step([(r, q[:n]) for r, q, n in zip(rids, seqs, lens)])
    for i in range(3):
        got[i].append(out[i:i + 1])
    for t in range(40):
        out = m.step([(r, [q[n + t]]) for r, q, n in zip(rids, seqs, lens)])
        for i in range(3):
            got[i].append(out[i:i + 1])
    assert m.graph_count() > 0
    for i, n in enumerate(lens):
        assert close(torch.cat(got[i]), want[i][n - 1:], dtype), i
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_greedy_generation_through_the_scheduler(dtype):
    """the framework's own entry points: generate() of the model and the continuous-batching scheduler; teacher-forced check of
    every generated token against the oracle's logits for the sequence the framework produced"""
    from pegainfer_b200.engine import Engine
    cfg = cfg_general()
    w = make_weights(cfg, 27)
    prompts = [tokens_for(cfg, n, 40 + n) for n in (5, 37, 1, 64, 18)]
    m = build(cfg, w, dtype, max_tokens=512, max_requests=3)
    outs = Engine(m).generate(prompts, 12, max_live=3, token_budget=48)
    alone, _, _ = m.generate(prompts[1], 12)
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        lg = oracle_logits(cfg, w, p + o[:-1])[len(p) - 1:].to(F32)
        top2 = lg.topk(2, -1).values
        gap_ok = (top2[:, 0] - top2[:, 1]) < (1e-3 if dtype == F32 else 0.15) * lg.std()
        assert ((lg.argmax(-1) == torch.tensor(o)) | gap_ok).all()
    if dtype == F32:
        assert alone == outs[1]
    m.close()


def test_checkpoint_folder_through_the_registry_and_the_trace_tool(tmp_path):
    import json
    import os
    import subprocess

    import numpy as np
    from safetensors.torch import save_file

    from pegainfer_b200.registry import architecture_of, load_model
    cfg = cfg_edges()
    w = make_weights(cfg, 28)
    for l in cfg["layers"]:
        l.pop("ranks", None)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    assert architecture_of(str(tmp_path)) == "Rilonex"
    m = load_model(str(tmp_path), "float32", max_tokens=256)
    toks = tokens_for(cfg, 40, 7)
    rid = m.alloc_request()
    want = oracle_logits(cfg, w, toks)
    assert close(m.step([(rid, toks)], [list(range(40))]), want, F32)
    m.close()
    # the same through the trace tool in a process of its own: two portions of one request beside a second request
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:25], "want": [0, 24]}, {"id": "b", "tokens": toks[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[25:], "want": [14]}, {"id": "b", "tokens": toks[3:9], "want": [5]}], "end": ["a", "b"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600,
                       env={k: v for k, v in os.environ.items() if not k.startswith("OMP_")} | {"PYTHONPATH": root})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1"]
    a0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1).copy())
    a1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1).copy())
    assert close(torch.cat([a0, a1]), want[[0, 24, 39, 8]], F32)
