"""Vegodra on the GPU against the plain oracle (oracle/vegodra_oracle.py): mechanisms alone through the C ABI or as one-layer
models, then the model through its own step / engine / generate entry points -- whole prompts, token-by-token decoding,
portions down to two tokens, unequal batches, reused pages and state slots, keys far back, at page and key-block borders and on
both sides of every chunk border, the first tokens, long decoding, greedy generation.

Configurations and weights are made here (small, random, seeded).  float32 runs are held to 2e-4 of the logits' spread
(against the oracle in fp64), bfloat16 runs to rounding noise.  Where random weights would blur a fault (one far key among
hundreds, a sink, a chunk's border) the inputs are built so that a single score dominates.
"""
import math
import random

import pytest
import torch

from oracle import vegodra_oracle as O

pytestmark = pytest.mark.gpu

F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16


# ------------------------------------------------------------------ configurations (none is a real checkpoint's)
def att(heads, kv_heads, dim, vdim, chunk, rot_dims, base=10000.0, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": {"dims": rot_dims, "base": base},
         "scale": scale if scale is not None else 1.5 / math.sqrt(dim)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=10000.0, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "rot": {"dims": rot_dim, "base": base}, "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}}


def gla(heads, dim, vdim, tau, rank):
    """'rank' only shapes the tensors; a checkpoint's config.json does not carry it"""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "rank": rank}


def model_cfg(layers, vocab=211, width=88, eps=1e-5):
    """layers: (mixer entry, hidden size of the feed-forward or 0)"""
    return {"architecture": "Vegodra", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(l, mlp={"kind": "dense", "ff": ff} if ff else None) for l, ff in layers]}


def cfg_general():
    """All sizes differ from each other; every mixer; a borrowing layer with another chunk and scale than the layer it reads, and more query
    heads per key head than rotate in the same way; a layer without feed-forward; tensor-core and generic attention kernels in bf16."""
    return model_cfg([(att(6, 3, 32, 32, 24, 12), 72), (lat(5, 24, 16, 40, 56, 64), 56), (gla(3, 20, 28, 9.0, 5), 0),
                      (att(6, 3, 32, 32, 40, 12, scale=0.11, kv_from=0), 104), (att(4, 2, 20, 36, 17, 8, base=300.0), 40), (lat(3, 18, 10, 14, 30, 48, base=500.0), 64),
                      (att(4, 2, 20, 36, 50, 8, base=300.0, kv_from=4), 0), (gla(2, 40, 12, 20.0, 16), 24)])


def cfg_edges():
    """Values that often coincide or equal one are made to differ or to be one: one head, kv_heads == heads, ranks of one, chunks of one token
    and of a page, tau of one, everything rotated, head sizes and widths that are no multiple of 4."""
    return model_cfg([(att(1, 1, 10, 7, 1, 10), 0), (gla(1, 9, 11, 1.0, 1), 19), (lat(1, 6, 2, 9, 1, 5), 33), (att(5, 5, 6, 6, 16, 2), 21),
                      (att(5, 5, 6, 6, 1000, 2, kv_from=3), 13), (lat(7, 11, 4, 6, 13, 21), 0), (gla(3, 7, 5, 0.5, 3), 0)], vocab=97, width=50, eps=1e-6)


def cfg_wide():
    """head sizes of the 128- and 256-wide register tiles, the widest tensor-core tiles, several layers reading one cache"""
    return model_cfg([(att(8, 2, 128, 128, 48, 64), 64), (gla(2, 128, 48, 16.0, 24), 40), (att(8, 2, 128, 128, 32, 64, kv_from=0), 0),
                      (lat(4, 64, 32, 48, 40, 192), 48), (gla(1, 160, 24, 5.0, 8), 0), (att(8, 2, 128, 128, 80, 64, kv_from=0), 32), (att(2, 1, 200, 256, 33, 100), 40)],
                     vocab=128, width=64)


CONFIGS = {"general": cfg_general, "edges": cfg_edges, "wide": cfg_wide}


def config_of(cfg):
    """the product's configuration object with the ranks filled in (as the loader does from the tensors' shapes)"""
    from pegainfer_b200.vegodra import VegodraConfig, with_ranks
    return with_ranks(VegodraConfig.from_dict(cfg), {f"l{i}.mix.a1": (l["rank"], cfg["width"]) for i, l in enumerate(cfg["layers"]) if "rank" in l})


def make_weights(cfg, seed, sharp=1.0):
    """bf16 checkpoint; `sharp` scales the latent attention's query factor so that single keys weigh far more than the rest (the other
    attention norms its queries and keys: its scale in the configuration does that)"""
    from pegainfer_b200.vegodra import weight_shapes
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in weight_shapes(config_of(cfg)).items():
        rn = lambda s=1.0: s * torch.randn(shape, generator=g)  # noqa: E731
        if name.endswith("mix.uq"):
            t = sharp * rn() / math.sqrt(shape[1])
        elif name.endswith((".norm", ".norm1")):
            t = 1.0 + rn(0.2)
        elif name.endswith(("norm.b", "norm1.b")):
            t = rn(0.3)
        elif name.endswith("a2.b"):
            t = 0.5 + rn(1.5)
        elif name.endswith("sink"):
            t = 0.5 + rn()
        elif name == "embed":
            t = 0.3 + 2 * rn()  # neither centred nor of unit size: the embedding's own norm shows
        else:
            t = rn() / math.sqrt(shape[-1])
        w[name] = t.to(BF16)
    return w


def build(cfg, w, dtype, max_tokens=1024, max_requests=4):
    from pegainfer_b200.vegodra import VegodraConfig, VegodraModel
    return VegodraModel(VegodraConfig.from_dict(cfg), w, dtype=dtype, max_tokens=max_tokens, max_requests=max_requests)


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
@pytest.mark.parametrize("W", [1, 50, 64, 4096, 13000])
@pytest.mark.parametrize("T", [1, 5, 90])
def test_layer_norm_steps(lib, dtype, W, T):
    """embedding with its own norm and the first layer's; residual sum with and without a norm after it; last norm over gathered rows.  The
    rows carry a large common offset: a variance that is not taken about the mean would show."""
    P = Hold()
    V, eps, f32 = 9, 1e-3, int(dtype == F32)
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    emb, y = rounded(30.0 + 0.1 * rnd(V, W), dtype), rounded(40.0 + rnd(T, W), dtype)
    w0, b0, w1, b1 = (rounded(c + 0.3 * rnd(W), dtype) for c in (1.0, 0.2, 1.0, -0.1))
    ids = [(3 * t + 1) % V for t in range(T)]
    x, h = torch.zeros(T, W, device="cuda"), torch.zeros(T, W, dtype=dtype, device="cuda")
    nxt = (P(dev(w1, dtype)), P(dev(b1, dtype)), h.data_ptr())
    tol = dict(atol=3e-5, rtol=1e-4) if dtype == F32 else dict(atol=4e-2, rtol=1e-2)
    assert lib.pk_res32_embed_lnorm(P(dev(emb, dtype)), P(i32(ids)), P(dev(w0, dtype)), P(dev(b0, dtype)), x.data_ptr(), *nxt, W, eps, T, f32, None) == 0
    torch.cuda.synchronize()
    ref = O.layer_norm(emb[ids].to(F64), w0, b0, eps)
    assert torch.allclose(x.cpu().to(F64), ref, atol=3e-4, rtol=1e-4)  # offsets of 30: the mean's own rounding
    assert torch.allclose(h.float().cpu().to(F64), O.layer_norm(ref, w1, b1, eps), atol=max(tol["atol"], 1e-3), rtol=tol["rtol"])
    x0 = rnd(T, W)
    x.copy_(x0)
    assert lib.pk_res32_add_lnorm(P(dev(y, dtype)), x.data_ptr(), *nxt, W, eps, T, f32, None) == 0
    torch.cuda.synchronize()
    ref = x0 + y
    assert torch.equal(x.cpu(), ref)
    want = O.layer_norm(ref.to(F64), w1, b1, eps)
    assert torch.allclose(h.float().cpu().to(F64), want, atol=max(tol["atol"], 1e-4), rtol=tol["rtol"])
    before = h.clone()
    assert lib.pk_res32_add_lnorm(P(dev(y, dtype)), x.data_ptr(), None, None, None, W, eps, T, f32, None) == 0
    rows = [T - 1, 0, 0]
    out = torch.zeros(3, W, dtype=dtype, device="cuda")
    assert lib.pk_res32_lnorm_rows(x.data_ptr(), P(i32(rows)), P(dev(w0, dtype)), P(dev(b0, dtype)), out.data_ptr(), W, eps, 3, f32, None) == 0
    torch.cuda.synchronize()
    assert torch.equal(before, h)
    want = O.layer_norm((ref + y).to(F64), w0, b0, eps)[rows]
    assert torch.allclose(out.float().cpu().to(F64), want, atol=max(tol["atol"], 2e-4), rtol=tol["rtol"])


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


def freq_table(rot):
    dims = rot["dims"]
    return (float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)).to(F32).cuda()


def run_attention(lib, dtype, mx, rows, sink, starts, lens, ps=16, max_kv=0, eps=1e-5, borrow=None):
    """norm + rotation + cache append + attention for a step whose request r brings positions starts[r] .. lens[r] - 1 (earlier positions
    were appended by a first call); rows [q | k | v | head gates].  borrow = (mixer, rows [q | head gates], sink): a second layer that reads the
    same cache.  Returns [T, H * vdim] (of the second layer when there is one)."""
    from pegainfer_b200.ffi import AttnExtra, QkPrep
    import ctypes as C
    P = Hold()
    G, D, Dv = mx["kv_heads"], mx["dim"], mx["vdim"]
    pages, off, n_pages = paged(lens, ps, shuffle_seed=5)
    stride = ps * G * (D + Dv) + 24
    cache = torch.full((n_pages, stride), float("nan"), dtype=dtype, device="cuda")  # a slot that nothing wrote must not be read
    f32 = int(dtype == F32)

    def layer(mx, rows, sink, rows_of, q_only):
        H, dims = mx["heads"], mx["rot"]["dims"]
        x = dev(torch.cat([rows[r][a:b] for r, (a, b) in enumerate(rows_of)]), dtype)
        p = [q for a, b in rows_of for q in range(a, b)]
        rq = [r for r, (a, b) in enumerate(rows_of) for _ in range(a, b)]
        T, ld, out_ld = len(p), x.shape[1], H * Dv + 6
        if T == 0:
            return None
        qo, out = torch.zeros(T, H * D, dtype=dtype, device="cuda"), torch.full((T, out_ld), 5.0, dtype=dtype, device="cuda")
        a = (P(i32(p)), P(i32(rq)), P(i32(off)), P(i32(pages)))
        prep = QkPrep(norm_kind=1, eps=eps, q_only=int(q_only))
        assert lib.pk_gqa_norm_append(P(x), ld, *a, qo.data_ptr(), None if q_only else cache.data_ptr(), stride, ps, H, G, D, Dv, dims, 0,
                                      P(freq_table(mx["rot"])) if dims else None, 1.0, C.byref(prep), T, f32, None) == 0
        gate_at = H * D + (0 if q_only else G * (D + Dv))
        ex = AttnExtra(gate=x.data_ptr() + gate_at * x.element_size(), gate_ld=ld, gate_per_head=1, out_ld=out_ld, max_kv_len=max_kv)
        assert lib.pk_gqa_attention_ex(qo.data_ptr(), cache.data_ptr(), P(dev(sink, dtype)) if sink is not None else None, *a, out.data_ptr(), stride, ps, T, H, G,
                                       D, Dv, float(mx["scale"]), mx["mask"]["size"], C.byref(ex), f32, None) == 0
        torch.cuda.synchronize()
        assert (out[:, H * Dv:] == 5.0).all()  # nothing past the heads' columns is written
        return out[:, :H * Dv].float().cpu()

    now = [(s, n) for s, n in zip(starts, lens)]
    layer(mx, rows, sink, [(0, s) for s in starts], False)
    got = layer(mx, rows, sink, now, False)
    return layer(borrow[0], borrow[1], borrow[2], now, True) if borrow else got


def oracle_attention(mx, x, sink, lo, hi, eps=1e-5, kv=None, cached=None):
    """The oracle's mechanisms on a stacked projection output, in fp64; what is cached is rounded to `cached`.  -> (rows lo .. hi - 1, (k, v))"""
    H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    x = x[:hi].to(F64)
    pos = torch.arange(hi)
    if kv is None:
        k = O.rms(O.rotate_halves(x[:, H * D:(H + G) * D].reshape(-1, G, D), pos, mx["rot"]), eps)
        kv = (rounded(k, cached).to(F64) if cached else k, x[:, (H + G) * D:(H + G) * D + G * Dv].reshape(-1, G, Dv))
        gate = x[:, (H + G) * D + G * Dv:]
    else:
        gate = x[:, H * D:]
    q = O.rms(O.rotate_halves(x[:, :H * D].reshape(-1, H, D), pos, mx["rot"]), eps)
    o = O.chunked_attention(q[lo:], kv[0], kv[1], mx, pos[lo:], sink.to(F64) if sink is not None else torch.full((H,), -1e30, dtype=F64))
    return (o * torch.sigmoid(gate[lo:, :H])[:, :, None]).flatten(1).to(F32), kv


# heads, kv heads, dim, vdim, rotated entries, chunk: bf16 with dim == vdim in (32, 64, 96, 128) runs on the tensor cores
ATTN_SHAPES = [(3, 1, 20, 12, 8, 33), (6, 2, 32, 32, 32, 64), (1, 1, 16, 16, 2, 1), (4, 4, 64, 64, 16, 100), (2, 1, 128, 128, 128, 48), (9, 3, 96, 96, 32, 0),
               (5, 5, 32, 32, 30, 7), (2, 2, 200, 256, 100, 130), (8, 2, 64, 64, 0, 128)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,Dv,dims,chunk", ATTN_SHAPES)
def test_attention_ragged_batch(lib, dtype, H, G, D, Dv, dims, chunk):
    """three requests in one launch: a 70-token portion that starts at position 90, one decoded token at position 199, and the first 5
    tokens of a sequence; with and without a sink and a known longest context; then a second layer with twice the heads, another chunk and
    scale that reads the same cache; a step of decoded tokens only"""
    g = torch.Generator().manual_seed(3)
    mx = att(H, G, D, Dv, chunk, dims, scale=2.0 / math.sqrt(D))["mixer"]
    mb = att(2 * H, G, D, Dv, chunk + 11 if chunk else 50, dims, scale=1.0 / math.sqrt(D))["mixer"]
    lens = [160, 200, 5]
    rows = [rounded(torch.randn(n, (H + G) * D + G * Dv + H, generator=g), dtype) for n in lens]
    rows_b = [rounded(torch.randn(n, 2 * H * D + 2 * H, generator=g), dtype) for n in lens]
    sink, sink_b = rounded(torch.randn(H, generator=g) + 1, dtype), rounded(torch.randn(2 * H, generator=g), dtype)
    tol = 4e-5 if dtype == F32 else 3e-2
    for starts in ([90, 199, 0], [159, 199, 4]):
        for (s, max_kv) in ((sink, 0), (sink, 200), (None, 200)):
            got = run_attention(lib, dtype, mx, rows, s, starts, lens, max_kv=max_kv)
            want = [oracle_attention(mx, rows[r], s, starts[r], lens[r], cached=dtype) for r in range(3)]
            assert (got - torch.cat([w for w, _ in want])).abs().max() < tol, (starts, max_kv)
        got = run_attention(lib, dtype, mx, rows, sink, starts, lens, max_kv=200, borrow=(mb, rows_b, sink_b))
        want = torch.cat([oracle_attention(mb, rows_b[r], sink_b, starts[r], lens[r], kv=kv)[0] for r, (_, kv) in enumerate(want)])
        assert (got - want).abs().max() < tol, starts


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("prompt", [False, True])
@pytest.mark.parametrize("H,D,chunk", [(2, 32, 64), (2, 24, 64), (3, 64, 48), (1, 128, 17), (2, 32, 600), (2, 64, 1)])
def test_single_keys_stand_out(lib, dtype, prompt, H, D, chunk):
    """Key and query of one pair point the same way and every other key at right angles to them, with a scale that leaves the rest no weight:
    the output must be that key's value when it lies in the query's chunk, and must not contain it when it lies one position before the
    chunk, one past the query, or far away.  Both sides of chunk, page (16) and key-block (64) borders, the first tokens, the query's own
    position.  `prompt`: the query sits in a 40-token portion, else it is a decoded token.  The sink is far below the aimed score."""
    mx = att(H, 1, D, D, chunk, 0, scale=30.0 / D)["mixer"]
    n = 700
    g = torch.Generator().manual_seed(4)
    val = rounded(torch.randn(n, D, generator=g), dtype)
    c0 = 690 // chunk * chunk
    cases = {(690, k) for k in (c0 - 2, c0 - 1, c0, c0 + 1, 0, 1, 15, 16, 63, 64, 300, 639, 640, 671, 672, 687, 688, 689, 690, 691)}
    for edge in (chunk, 2 * chunk, 5 * chunk):
        if edge < n - 2:
            cases |= {(edge - 1, edge - 1), (edge - 1, edge - chunk), (edge, edge - 1), (edge, edge), (edge + 1, edge), (edge + 1, edge - 1)}
    cases |= {(0, 0), (1, 0), (1, 1), (2, 1), (15, 16), (16, 15)}
    sink = torch.full((H,), -5.0)
    for q_at, kp in sorted(c for c in cases if c[1] >= 0):
        rows = torch.zeros(n, H * D + 2 * D + H)
        rows[:, H * D + 1] = 1.0                    # every key along entry 1 ...
        rows[kp, H * D], rows[kp, H * D + 1] = 1.0, 0.0  # ... the aimed one along entry 0
        rows[:, H * D + D:H * D + 2 * D] = val
        rows[:, H * D + 2 * D:] = 20.0              # gates wide open
        for h in range(H):
            rows[:, h * D] = 1.0                    # every query asks along entry 0
        hi = max(q_at, kp) + 1
        start = max(q_at - 39, 0) if prompt else q_at
        got = run_attention(lib, dtype, mx, [rounded(rows, dtype)], sink, [start], [hi], max_kv=hi)[q_at - start]
        seen = kp <= q_at and kp // chunk == q_at // chunk
        lo = q_at // chunk * chunk
        own = val[lo:q_at + 1].to(F64)
        if seen:
            want = val[kp]
        else:  # all visible keys weigh the same, the sink e^-5 of one of them
            want = (own.sum(0) / (q_at + 1 - lo + math.exp(-5.0))).to(F32)
        for h in range(H):
            assert torch.allclose(got[h * D:(h + 1) * D], want, atol=2e-2, rtol=1e-2), (q_at, kp, h)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", [32, 20])
@pytest.mark.parametrize("T", [1, 40])
def test_sink_counts_once_and_is_not_scaled(lib, dtype, D, T):
    """equal scores of zero over a chunk and sinks of ln 3 and 50: the output is the values' sum over (number of keys + 3), and nothing"""
    mx = att(2, 1, D, D, 64, 0, scale=7.0)["mixer"]
    n = 40
    rows = torch.zeros(n, 4 * D + 2)
    val = rounded(torch.randn(n, D, generator=torch.Generator().manual_seed(8)), dtype)
    rows[:, 3 * D:4 * D] = val
    rows[:, 4 * D] = 20.0
    sink = torch.tensor([math.log(3.0), 50.0])
    got = run_attention(lib, dtype, mx, [rounded(rows, dtype)], sink, [n - T], [n], max_kv=n)
    s = rounded(sink, dtype)
    for i in range(T):
        k = n - T + i + 1
        assert torch.allclose(got[i, :D], val[:k].sum(0) / (k + s[0].exp()), atol=1e-5 if dtype == F32 else 1e-2)
    assert got[:, D:].abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T", [1, 6, 9, 50])
@pytest.mark.parametrize("H,D,R,rank,q_rank,dims", [(3, 20, 10, 24, 14, 10), (4, 64, 16, 64, 48, 16), (2, 7, 4, 9, 1, 2), (5, 32, 64, 192, 600, 64), (2, 16, 8, 1000, 1100, 8)])
def test_latent_norms_append_and_query(lib, dtype, T, H, D, R, rank, q_rank, dims):
    """the queries' latent and the cached latent are normed with their own weights, the shared key part and the queries rotate neighbouring
    entries, the unrotated query is folded onto the latent"""
    P = Hold()
    g = torch.Generator().manual_seed(6)
    ps, eps, f32, n0 = 8, 1e-3, int(dtype == F32), 75
    rnd = lambda *s: rounded(torch.randn(*s, generator=g), dtype)  # noqa: E731
    ld, q_off, kv_off = q_rank + rank + R + 9, 3, q_rank + 5
    rows, wq, wk = 0.05 * rnd(T, ld), rounded(1 + 0.3 * torch.randn(q_rank, generator=g), dtype), rounded(1 + 0.3 * torch.randn(rank, generator=g), dtype)
    rows = rounded(rows, dtype)
    pos = torch.arange(n0, n0 + T)
    pages, off, n_pages = paged([n0 + T], ps)
    stride = ps * (rank + R) + 8
    cache, cq = torch.full((n_pages, stride), 9.0, dtype=dtype, device="cuda"), torch.zeros(T, q_rank, dtype=dtype, device="cuda")
    rot = {"dims": dims, "base": 800.0}
    fr = freq_table(rot)
    where = (P(i32(pos.tolist())), P(i32([0] * T)), P(i32(off)), P(i32(pages)))
    assert lib.pk_latent_prep(P(dev(rows, dtype)), ld, q_off, q_rank, P(dev(wq, dtype)), cq.data_ptr(), kv_off, P(dev(wk, dtype)), *where, cache.data_ptr(), stride, ps,
                              rank, R, dims, 1, fr.data_ptr(), 1.0, eps, T, f32, None) == 0
    q, uk = rnd(T, H, D + R), rnd(H, D, rank)
    qa = torch.zeros(T, H, rank + R, dtype=dtype, device="cuda")
    assert lib.pk_latent_query(P(dev(q, dtype)), P(dev(uk.transpose(1, 2), dtype)), qa.data_ptr(), where[0], T, H, D, rank, R, dims, 1, fr.data_ptr(), 1.0, f32,
                               None) == 0
    torch.cuda.synchronize()
    x = rows.to(F64)
    tol = dict(atol=3e-5, rtol=1e-4) if dtype == F32 else dict(atol=2e-2, rtol=1e-2)
    assert torch.allclose(cq.float().cpu().to(F64), O.rms(x[:, q_off:q_off + q_rank], eps) * wq, **tol)
    want = torch.cat([O.rms(x[:, kv_off:kv_off + rank], eps) * wk, O.rotate_neighbours(x[:, None, kv_off + rank:kv_off + rank + R], pos, rot)[:, 0]], 1)
    c = cache.float().cpu()
    got = torch.stack([c[pages[int(p) // ps], int(p) % ps * (rank + R):(int(p) % ps + 1) * (rank + R)] for p in pos])
    assert torch.allclose(got.to(F64), want, **tol)
    assert (c == 9.0).sum().item() == c.numel() - got.numel() + (got == 9.0).sum().item()
    qd = q.to(F64)
    want = torch.cat([torch.einsum("thd,hdr->thr", qd[..., :D], uk.to(F64)), O.rotate_neighbours(qd[..., D:], pos, rot)], -1)
    assert torch.allclose(qa.float().cpu().to(F64), want, atol=2e-4 if dtype == F32 else 6e-2, rtol=1e-4 if dtype == F32 else 1e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rank,R", [(64, 16), (48, 6), (192, 32)])
@pytest.mark.parametrize("prompt", [False, True])
def test_latent_attention_finds_far_keys(lib, dtype, rank, R, prompt):
    """one position among 1500 is aimed at through the latent part alone, another through the shared rotated part alone: no window, no sink"""
    P = Hold()
    n, H, ps, f32 = 1500, 3, 16, int(dtype == F32)
    g = torch.Generator().manual_seed(7)
    c = rounded(0.3 * torch.randn(n, rank + R, generator=g), dtype)
    pages, off, n_pages = paged([n], ps, 3)
    stride = ps * (rank + R)
    cache = torch.full((n_pages, ps, rank + R), float("nan"))
    for p in range(n):
        cache[pages[p // ps], p % ps] = c[p]
    for q_at, kp in ((1499, 0), (1499, 1), (1499, 15), (1499, 16), (1499, 64), (1499, 700), (1499, 1498), (1499, 1499), (640, 639), (640, 641), (63, 63), (0, 0)):
        for part in (slice(0, rank), slice(rank, rank + R)):
            start = max(q_at - 40, 0) if prompt else q_at
            T = q_at + 1 - start
            aim = torch.zeros(rank + R)
            aim[part] = c[kp, part] / c[kp, part].norm() ** 2
            qa = rounded(aim.expand(T, H, -1) * 60.0, dtype)
            out = torch.zeros(T, H, rank, dtype=dtype, device="cuda")
            assert lib.pk_latent_attention_ex(P(dev(qa, dtype)), P(dev(cache, dtype)), None, P(i32(list(range(start, q_at + 1)))), P(i32([0] * T)), P(i32(off)),
                                              P(i32(pages)), out.data_ptr(), stride, ps, T, H, rank, R, 1.0, 0, q_at + 1, f32, None) == 0
            torch.cuda.synchronize()
            s = (qa[-1, 0].to(F64) @ c[:q_at + 1].to(F64).T).softmax(-1)
            want = (s @ c[:q_at + 1, :rank].to(F64)).to(F32)
            assert torch.allclose(out[-1].float().cpu(), want.expand(H, -1), atol=2e-5 if dtype == F32 else 2e-2), (q_at, kp, part)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows", [1, 8, 20, 70])
@pytest.mark.parametrize("batch,cols,K", [(3, 40, 24), (5, 14, 7), (1, 130, 64), (4, 33, 16)])
def test_batched_product_with_element_gate(lib, dtype, rows, batch, cols, K):
    P = Hold()
    g = torch.Generator().manual_seed(11)
    lda, ldc, ldg = batch * K + 8, batch * cols + 6, batch * cols + 5
    A, B, Z = (rounded(torch.randn(*s, generator=g), dtype) for s in ((rows, lda), (batch, cols, K), (rows, ldg)))
    out = torch.full((rows, ldc), 7.0, dtype=dtype, device="cuda")
    z = dev(Z, dtype)
    assert lib.pk_gemm_strided_gated(P(dev(A, dtype)), P(dev(B, dtype)), out.data_ptr(), z.data_ptr() + 2 * z.element_size(), rows, cols, K, lda, K, ldc, batch, K,
                                     cols * K, cols, ldg, cols, int(dtype == F32), None) == 0
    torch.cuda.synchronize()
    want = torch.einsum("rbk,bck->rbc", A[:, :batch * K].reshape(rows, batch, K), B).reshape(rows, -1) * torch.sigmoid(Z[:, 2:2 + batch * cols])
    assert torch.allclose(out.float().cpu()[:, :batch * cols], want, atol=1e-4 if dtype == F32 else 3e-2, rtol=1e-4 if dtype == F32 else 1e-2)
    assert (out[:, batch * cols:] == 7.0).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,Dv,tau", [(3, 20, 24, 16.0), (4, 32, 48, 1.0), (2, 64, 100, 0.5), (2, 128, 16, 30.0), (1, 200, 8, 7.0), (5, 9, 3, 4.0)])
def test_gated_linear_attention_in_portions_over_reused_slots(lib, dtype, H, D, Dv, tau):
    """two sequences advance in portions of 1, 37, 2 and 150 tokens through slots 2 and 0; decays from nearly zero to nearly one; every other
    step with the decays made by a launch of their own"""
    P = Hold()
    g = torch.Generator().manual_seed(10)
    lens = [190, 260]
    Cn = 2 * H * D + H * Dv
    ld, ldc = Cn + 8, H * D + 1
    xs = [rounded(torch.randn(n, Cn, generator=g), dtype) for n in lens]
    zs = [4 * torch.randn(n, ldc, generator=g) for n in lens]
    bias = torch.randn(H * D, generator=g)
    want = []
    for x, z in zip(xs, zs):
        x, z = x.to(F64), z.to(F64)
        q, k, v = x[:, :H * D].reshape(-1, H, D) * D ** -0.5, x[:, H * D:2 * H * D].reshape(-1, H, D), x[:, 2 * H * D:].reshape(-1, H, Dv)
        o, _ = O.decayed_memory(q, k, v, O.channel_decay(z[:, :H * D] + bias, tau).reshape(-1, H, D))
        want.append(o.flatten(1).to(F32))
    stride = H * D * Dv + 11
    state = torch.zeros(3, stride, device="cuda")
    slots, at, got = [2, 0], [0, 0], [[], []]
    sizes, k = [1, 37, 2, 150], 0
    while any(at[r] < lens[r] for r in range(2)):
        live = [r for r in range(2) if at[r] < lens[r]]
        ns = [min(sizes[(k + r) % 4], lens[r] - at[r]) for r in live]
        T = sum(ns)
        cut = lambda src: torch.cat([src[r][at[r]:at[r] + m] for r, m in zip(live, ns)])  # noqa: E731
        rows = torch.zeros(T, ld)
        rows[:, 8:] = cut(xs)
        row0 = [sum(ns[:e]) for e in range(len(ns))]
        out = torch.zeros(T, H * Dv, device="cuda")
        z_d, ready = cut(zs).cuda(), k % 2
        if ready:
            z_d = z_d[:, :H * D].contiguous()
            assert lib.pk_logistic_decay(P(z_d), P(bias.cuda()), tau, T, H * D, None) == 0
        assert lib.pk_gla_seq(P(dev(rows, dtype)), ld, 8, 8 + H * D, 8 + 2 * H * D, P(z_d), z_d.shape[1], ready, P(bias.cuda()), tau, state.data_ptr(), stride,
                              P(i32([slots[r] for r in live])), P(i32(row0)), P(i32(ns)), out.data_ptr(), H, D, Dv, len(ns), int(dtype == F32), None) == 0
        torch.cuda.synchronize()
        o = out.cpu()
        for e, (r, m) in enumerate(zip(live, ns)):
            got[r].append(o[row0[e]:row0[e] + m])
            at[r] += m
        k += 1
    for r in range(2):
        assert torch.allclose(torch.cat(got[r]), want[r], atol=1e-4, rtol=1e-4), r
    assert state[1].abs().max().item() == 0.0 and state[:, H * D * Dv:].abs().max().item() == 0.0  # nothing outside the owned blocks is touched


@pytest.mark.parametrize("T", [1, 4, 9, 300])
@pytest.mark.parametrize("W,ff,ld", [(64, 96, 136), (256, 520, 520), (128, 72, 75)])
def test_gate_and_up_projection_with_gelu_in_the_epilogue(lib, T, W, ff, ld):
    """rows of their own stride; the tanh form, which differs from the exact one by more than the tolerance used here in fp32"""
    from pegainfer_b200.ffi import GemvArgs
    import ctypes as C
    P = Hold()
    g = torch.Generator().manual_seed(13)
    x, wt = rounded(torch.randn(T, W, generator=g), BF16), rounded(2 * torch.randn(2 * ff, W, generator=g) / math.sqrt(W), BF16)
    gate, up = rounded(x @ wt[:ff].T, BF16), rounded(x @ wt[ff:].T, BF16)
    want = O.gelu_tanh(gate) * up
    for dtype in (F32, BF16):
        two = torch.full((T, ld), 6.0, dtype=dtype, device="cuda")
        assert lib.pk_act_ex(P(dev(torch.cat([gate, up], 1), dtype)), two.data_ptr(), ld, ff, T, 3, int(dtype == F32), None) == 0
        torch.cuda.synchronize()
        assert torch.allclose(two[:, :ff].float().cpu(), want, atol=1e-5 if dtype == F32 else 1e-3, rtol=1e-5 if dtype == F32 else 1e-2)
        assert (two[:, ff:] == 6.0).all()
    out = torch.full((T, ld), 6.0, dtype=BF16, device="cuda")
    if T <= 4:
        a = GemvArgs()
        a.W, a.X, a.M, a.N, a.K, a.epi, a.y_ld = P(dev(wt, BF16)), P(dev(x, BF16)), ff, T, W, 6, ld
        a.Y[0], a.seg_rows[0] = out.data_ptr(), ff
        assert lib.pk_b200_gemv_fused(C.byref(a), None) == 0
    else:
        rc = lib.pk_b200_gemm_gated_ex(P(dev(wt, BF16)), P(dev(x, BF16)), out.data_ptr(), ff, T, W, ld, 2, None)
        if rc == -2:
            pytest.skip("shape outside the fused kernel's range (the host then runs two launches)")
        assert rc == 0
    torch.cuda.synchronize()
    assert torch.allclose(out[:, :ff].float().cpu(), want, atol=3e-2, rtol=3e-2)
    assert (out[:, ff:] == 6.0).all()


# ------------------------------------------------------------------ one-layer models: each mixer and the feed-forward alone
ONE = {"attention": (att(4, 2, 32, 32, 20, 16), 0), "attention_generic": (att(4, 4, 18, 24, 20, 6), 0), "latent": (lat(4, 32, 16, 24, 40, 64), 0),
       "latent_generic": (lat(3, 20, 6, 24, 22, 36), 0), "gla": (gla(4, 20, 12, 10.0, 6), 0), "mlp": (gla(1, 4, 4, 10.0, 2), 60)}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("which", sorted(ONE))
def test_each_mechanism_alone(dtype, which):
    """a portion, then decoded tokens; the sublayer's output projection is large, so that its result dominates the residual"""
    cfg = model_cfg([ONE[which]], vocab=64, width=48)
    w = make_weights(cfg, 14, SHARP[dtype])
    out = "l0.mlp.down" if which == "mlp" else "l0.mix.o"
    w[out] = (4.0 * w[out].float()).to(BF16)
    if which == "mlp":
        w["l0.mix.o"] = torch.zeros_like(w["l0.mix.o"])
    toks = tokens_for(cfg, 90, 3)
    m = build(cfg, w, dtype)
    rid = m.alloc_request()
    got = torch.cat([m.step([(rid, toks[:50])], [list(range(50))])] + [m.step([(rid, [t])]) for t in toks[50:]])
    assert close(got, oracle_logits(cfg, w, toks), dtype)
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_rows_of_the_order_of_sqrt_eps(dtype):
    """projections shrunk so that the eps of the heads' norms, of the latents' norms and of the read-out norm shows in the result; the
    embedding shrunk so that the layer norm's does"""
    cfg = model_cfg([(att(2, 1, 12, 16, 30, 6, scale=1.0), 0), (lat(2, 12, 4, 16, 10, 20), 0), (gla(2, 12, 8, 8.0, 4), 0)], vocab=64, width=48, eps=1e-3)
    w = make_weights(cfg, 15)
    for n in ("l0.mix.q", "l0.mix.k", "l1.mix.dq", "l1.mix.dkv", "l2.mix.v", "embed"):
        w[n] = (w[n].float() * 3e-2).to(BF16)
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
@pytest.mark.parametrize("sizes", [(2,), (3, 2, 16, 1, 37, 5), (64, 2, 2), (33, 1), (24,)])
def test_prompt_in_portions(name, dtype, sizes):
    """portions cut anywhere (inside pages, key blocks and chunks, and at a chunk's edge), down to two tokens"""
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
        h = r.choice([1, 2, 3, 4, 6, 8, 10])
        return h, r.choice([d for d in range(1, h + 1) if h % d == 0])
    layers, owners = [], []
    for i in range(r.randint(2, 7)):
        kind = r.choice(["attention", "attention", "latent", "gla"])
        if kind == "attention" and owners and r.random() < 0.5:
            j = r.choice(owners)
            o = layers[j][0]["mixer"]
            l = att(o["heads"], o["kv_heads"], o["dim"], o["vdim"], r.choice([1, 5, 16, 31, 64, 200]), o["rot"]["dims"], o["rot"]["base"], r.uniform(0.05, 0.5), kv_from=j)
        elif kind == "attention":
            h, g = heads()
            d = r.choice([8, 12, 16, 20, 32, 48, 64])
            l = att(h, g, d, r.choice([8, 16, 28, d, d]), r.choice([1, 3, 16, 24, 50, 64, 300]), r.choice([2, d // 2 // 2 * 2, d]), r.choice([100.0, 10000.0, 500000.0]),
                    r.uniform(0.05, 0.5))
            owners.append(i)
        elif kind == "latent":
            l = lat(heads()[0], r.choice([8, 12, 20, 32, 48]), r.choice([2, 6, 16, 32]), r.choice([8, 16, 28, 40]), r.choice([1, 8, 14, 40]),
                    r.choice([8, 20, 64, 128]), r.choice([100.0, 10000.0, 500000.0]), r.uniform(0.05, 0.4))
        else:
            l = gla(heads()[0], r.choice([4, 8, 12, 20, 32, 40, 72, 130]), r.choice([4, 8, 16, 28, 48]), r.choice([1.0, 4.0, 16.0, 25.0]), r.choice([1, 6, 8, 16, 24]))
        layers.append((l, r.choice([0, 8, 20, 56, 88])))
    return model_cfg(layers, vocab=r.randint(40, 300), width=r.choice([24, 36, 41, 64, 100]), eps=r.choice([1e-5, 1e-6, 1e-3]))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("seed", range(20))
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


def test_a_request_may_pause_while_others_go_on():
    """a request left out of some steps continues from its own cache and state"""
    cfg = cfg_general()
    w = make_weights(cfg, 31)
    a, b = tokens_for(cfg, 60, 1), tokens_for(cfg, 70, 2)
    m = build(cfg, w, F32, max_tokens=256, max_requests=2)
    ra, rb = m.alloc_request(), m.alloc_request()
    got_a, got_b = [], []
    for ea, eb in ((20, 30), (0, 5), (0, 1), (7, 1), (0, 33), (33, 0)):
        entries = ([(ra, a[len(got_a):len(got_a) + ea])] if ea else []) + ([(rb, b[len(got_b):len(got_b) + eb])] if eb else [])
        out = m.step(entries, [list(range(len(t))) for _, t in entries])
        got_a += list(out[:ea])
        got_b += list(out[ea:])
    assert close(torch.stack(got_a), oracle_logits(cfg, w, a), F32) and close(torch.stack(got_b), oracle_logits(cfg, w, b), F32)
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


def test_inconsistent_layers_are_refused():
    for bad in ([(att(2, 1, 8, 8, 4, 4, kv_from=0), 0)], [(att(2, 1, 8, 8, 4, 4), 0), (att(2, 2, 8, 8, 4, 4, kv_from=0), 0)],
                [(gla(1, 4, 4, 2.0, 2), 0), (att(2, 1, 8, 8, 4, 4, kv_from=0), 0)], [(att(2, 1, 300, 8, 4, 4), 0)], [(att(3, 2, 8, 8, 4, 4), 0)]):
        cfg = model_cfg(bad, vocab=30, width=16)
        with pytest.raises(RuntimeError):
            build(cfg, make_weights(cfg, 1), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_and_captured_steps(dtype):
    """a 300-token prompt and 260 decoded tokens (captured launch sequences from the second step of a kind on, across chunk edges and a graph
    bucket border at 512) against the same steps run eagerly and against the oracle"""
    cfg = model_cfg([(att(4, 2, 32, 32, 110, 16), 32), (lat(2, 24, 16, 20, 18, 64), 0), (gla(2, 16, 16, 30.0, 3), 40), (att(4, 2, 32, 32, 256, 16, kv_from=0), 24)],
                    vocab=96, width=64)
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
        l.pop("rank", None)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    assert architecture_of(str(tmp_path)) == "Vegodra"
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
