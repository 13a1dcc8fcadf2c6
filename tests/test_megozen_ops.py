"""Each mechanism of Megozen alone, against its plain statement: on the CPU and, marked gpu, the kernels in fp32 and bf16,
with sizes that hit and miss their vector and tensor-core paths."""
import math

import pytest
import torch

import plain_megozen as plain
from easyllm_b200.ops import infer as iops
from test_pafodra_ops import BF16, DEVICES, F32, _device, close, meta_of, rand


def tol(dtype, fp32=3e-6, bf16=2e-2):
    return fp32 if dtype == F32 else bf16


# ---- embedding ---------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,vocab,buckets,mp,mc", [(64, 50, 13, 7, 3), (37, 9, 1, 5, 2), (256, 300000, 499979, 90001, 70003)])
def test_pair_embedding_with_and_without_a_history(device, dtype, W, vocab, buckets, mp, mc):
    dev = _device(device)
    if vocab > 1000:
        W = 8
    table, pairs = rand(vocab, W, seed=1).to(dtype).to(dev), rand(buckets + 1, W, seed=2).to(dtype).to(dev)
    w = {"embed": table.double().cpu(), "bigram": pairs.double().cpu()}
    cfg = {"embedding": {"bigram": dict(buckets=buckets, mul_prev=mp, mul_cur=mc)}}
    g = torch.Generator().manual_seed(3)
    seqs = [torch.randint(0, vocab, (n,), generator=g).tolist() for n in (7, 1, 12)]
    want = [plain.embed(cfg, w, s) for s in seqs]
    ids = torch.tensor(sum(seqs, []), device=dev)
    got = iops.embed_pairs(ids, table, pairs, 1.0, mp, mc, meta_of([len(s) for s in seqs], dev))
    close(got, torch.cat(want), 1e-6)
    # the same sequences in pieces over their slots; a slot's old entries do not reach a sequence that starts
    hist = torch.full((4, 16), vocab - 1, dtype=torch.int32, device=dev)
    slots, at, out = [2, 0, 3], [0, 0, 0], [[], [], []]
    for piece in (4, 2, 1, 5):
        live = [i for i in range(3) if at[i] < len(seqs[i])]
        n = [min(piece, len(seqs[i]) - at[i]) for i in live]
        place = [(slots[i] * 16, at[i] + j + 1) for i, c in zip(live, n) for j in range(c)]
        m = meta_of(n, dev)
        m["kv_base"], m["kv_len"] = (torch.tensor(x, dtype=torch.int32, device=dev) for x in zip(*place))
        step = torch.tensor(sum((seqs[i][at[i]:at[i] + c] for i, c in zip(live, n)), []), device=dev)
        for i, o in zip(live, iops.embed_pairs(step, table, pairs, 1.0, mp, mc, m, hist).split(n)):
            out[i].append(o)
            at[i] += o.shape[0]
    for o, x in zip(out, want):
        close(torch.cat(o), x, 1e-6)


# ---- norms -------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,W", [(1, 8), (5, 100), (3, 1024), (2, 1028), (4, 4096), (2, 7000), (2, 8196), (3, 37)])
def test_two_layer_norms_of_one_row(device, dtype, n, W):
    dev = _device(device)
    x, w1, w2 = rand(n, W, seed=1) * 3 + 5, rand(W, seed=2), rand(W, seed=3)
    a, b = iops.layer_norms(x.to(dev), [w1.to(dev), w2.to(dev)], 1e-4, dtype)
    close(a, plain.layer_norm(x.double(), w1.double(), 1e-4), tol(dtype, bf16=8e-3))
    close(b, plain.layer_norm(x.double(), w2.double(), 1e-4), tol(dtype, bf16=8e-3))
    close(iops.layer_norms(x.to(dev), [w2.to(dev)], 0.5, dtype)[0], plain.layer_norm(x.double(), w2.double(), 0.5),
          tol(dtype, bf16=8e-3))


# ---- rotation ------------------------------------------------------------------------------------
ROTS = [dict(dims=16, base=10000.0), dict(dims=32, base=250.0, scaling=dict(factor=8.0, original=64, fast=8.0, slow=0.5)),
        dict(dims=8, base=1e6, scaling=dict(factor=2.5, original=4096, fast=32.0, slow=1.0)),
        dict(dims=4, base=50.0, scaling=dict(factor=1.0, original=10, fast=1.0, slow=1.0)),
        dict(dims=64, base=1e4, scaling=dict(factor=40.0, original=2, fast=1e9, slow=1e-9))]


@pytest.mark.parametrize("r", ROTS)
def test_rotary_tables_follow_the_scaled_frequencies(r):
    from easyllm_b200.models.layers import YarnRotaryTables
    tables = YarnRotaryTables(r["dims"], r["base"], r.get("scaling"))
    f, m = plain.frequencies(r)
    for need in (3, 5000):
        cos, sin = tables.get(need, torch.device("cpu"))
        assert cos.shape[0] >= need and cos.dtype == F32
        for p in (0, 1, 2, need - 1):
            for i, fi in enumerate(f):
                assert abs(float(cos[p, i]) - math.cos(p * fi) * m) < 2e-7 * m
                assert abs(float(sin[p, i]) - math.sin(p * fi) * m) < 2e-7 * m


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,dim,rt,rank,dims", [(4, 32, 16, 48, 16), (3, 10, 6, 13, 4), (1, 5, 2, 7, 2), (16, 128, 64, 512, 64),
                                                (2, 8, 24, 8, 16), (5, 8, 64, 1200, 32)])
@pytest.mark.parametrize("separate", [False, True])
def test_rotations_latent_norm_and_cache_rows(device, dtype, H, dim, rt, rank, dims, separate):
    from easyllm_b200.models.layers import YarnRotaryTables
    dev = _device(device)
    n, r = 6, dict(dims=dims, base=100.0, scaling=dict(factor=4.0, original=32, fast=4.0, slow=0.5))
    at = H * (dim + rt)
    z0 = rand(n, at + rank + rt + H, seed=1).to(dtype)
    w = rand(rank, seed=2) + 1
    pos = [0, 1, 7, 300, 301, 2]
    cos, sin = YarnRotaryTables(dims, 100.0, r["scaling"]).get(302, dev)
    m = dict(position_ids=torch.tensor(pos, dtype=torch.int32, device=dev),
             kv_base=torch.tensor([0, 0, 400, 400, 400, 800], dtype=torch.int32, device=dev),
             kv_len=torch.tensor([p + 1 for p in pos], dtype=torch.int32, device=dev))
    ld = -(-(rank + rt) // 8) * 8
    cache = torch.zeros(3, 400, ld, dtype=dtype, device=dev)
    z = z0.clone().to(dev)
    q = torch.zeros(n, H, 16 + rt, dtype=dtype, device=dev) if separate else None
    iops.latent_inputs(z, H, dim, rt, rank, w.to(dev), 1e-3, cos, sin, m, cache, None if q is None else q[..., 16:])
    z0d = z0.double()
    q_want = plain.rotate(z0d[:, :at].view(n, H, dim + rt)[..., dim:], pos, r)
    c_want = plain.rms_norm(z0d[:, at:at + rank], w.double(), 1e-3)
    k_want = plain.rotate(z0d[:, at + rank:at + rank + rt], pos, r)
    zq = z[:, :at].reshape(n, H, dim + rt)
    close(zq[..., dim:] if q is None else q[..., 16:], q_want, tol(dtype, bf16=8e-3))
    assert torch.equal(zq[..., :dim].cpu(), z0[:, :at].view(n, H, dim + rt)[..., :dim])
    if q is not None:
        assert torch.equal(zq.cpu(), z0[:, :at].view(n, H, dim + rt)) and float(q[..., :16].abs().max()) == 0
    close(z[:, at:at + rank], c_want, tol(dtype, bf16=8e-3))
    close(z[:, at + rank:at + rank + rt], k_want, tol(dtype, bf16=8e-3))
    assert torch.equal(z[:, at + rank + rt:].cpu(), z0[:, at + rank + rt:])
    rows = cache.view(-1, ld)[(m["kv_base"] + m["kv_len"] - 1).long()]
    assert torch.equal(rows[:, :rank + rt], z[:, at:at + rank + rt])
    assert int((cache.view(-1, ld).abs().sum(-1) > 0).sum()) == n


# ---- attention -----------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,d,dv,window", [(4, 64, 48, 40), (16, 576, 512, 130), (20, 80, 64, None), (33, 184, 144, 64), (1, 24, 16, 1),
                                           (3, 19, 13, 7), (40, 104, 40, 65)])
@pytest.mark.parametrize("gated", [False, True])
def test_attention_in_the_latent_space(device, dtype, H, d, dv, window, gated):
    """Decoding and continued rows over a cache: far keys, keys just inside and just outside the window, tile borders."""
    dev = _device(device)
    N, slot_rows = 300, 320
    scale = 0.6 / math.sqrt(d)
    keys = [rand(N, d, seed=s).to(dtype) for s in (1, 2)]
    places = [(0, 0), (0, 63), (0, 64), (0, 65), (0, 128), (1, 129), (0, 255), (1, 256), (0, 299), (1, 191), (1, 1)]
    q = rand(len(places), H, d, seed=3)
    W = window or 10 ** 9
    for row, (s, i) in enumerate(places):                 # the edge of the window, one past it, the first key, itself
        for h, j in enumerate((i - W + 1, i - W, 0, i)):
            if 0 <= j <= i and h < H:
                q[row, h] = 0.3 * q[row, h] + 12 / scale * keys[s][j].float() / keys[s][j].float().norm() ** 2
    q = q.to(dtype)
    g = rand(len(places), H + 3, seed=4).to(dtype)
    ld = -(-d // 8) * 8
    cache = rand(3, slot_rows, ld, seed=9).to(dtype)
    slots = (2, 0)
    for s in (0, 1):
        cache[slots[s], :N, :d] = keys[s]
    seen = [keys[s][max(0, i - W + 1):i + 1].double()[:, None].expand(-1, H, -1) for s, i in places]
    want = torch.stack([plain.attend(q[row].double(), k, k[..., :dv], scale) for row, k in enumerate(seen)])
    if gated:
        want = want * plain.sigmoid(g[:, 2:2 + H].double())[..., None]
    base = torch.tensor([slots[s] * slot_rows for s, _ in places], dtype=torch.int32, device=dev)
    n = torch.tensor([i + 1 for _, i in places], dtype=torch.int32, device=dev)
    gd = g.to(dev)[:, 2:2 + H] if gated else None
    for rows in (range(len(places)), [8], [0, 8]):        # one row alone is split over many ranges of keys
        rows = list(rows)
        got = iops.attention_latent(q[rows].to(dev), cache.to(dev).view(-1, ld), dv, base[rows].contiguous(), n[rows].contiguous(),
                                    int(max(n[rows])), scale, window, gd[rows] if gated else None)
        close(got, want[rows], tol(dtype, 1e-5, 1.5e-2))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M", [1, 8, 9, 40])
@pytest.mark.parametrize("H,N,K,ld", [(4, 48, 32, 48), (3, 13, 10, 16), (16, 512, 128, 192), (2, 8, 96, 96)])
def test_products_per_head(device, dtype, M, H, N, K, ld):
    dev = _device(device)
    x, w = rand(M, H, ld, seed=1).to(dtype).to(dev), rand(H, N, K, seed=2, scale=K ** -0.5).to(dtype).to(dev)
    want = torch.einsum("thk,hnk->thn", x.double().cpu()[..., :K], w.double().cpu())
    out = torch.zeros(M, H, N + 8, dtype=dtype, device=dev)
    iops.head_products(x[..., :K], w, out[..., :N])
    close(out[..., :N], want, tol(dtype, bf16=8e-3))
    assert float(out[..., N:].abs().max()) == 0
    close(iops.head_products(x[..., :K], w), want, tol(dtype, bf16=8e-3))


@pytest.mark.gpu
@pytest.mark.parametrize("H,dim,rt,rank,dv", [(4, 32, 16, 48, 24), (3, 64, 64, 64, 64), (2, 128, 64, 64, 128), (2, 8, 8, 16, 8),
                                              (2, 72, 40, 24, 96)])
@pytest.mark.parametrize("counts,window", [([300], 64), ([300], 100), ([5, 257, 130], 129), ([520], None), ([40, 1, 200], 1),
                                           ([600], 128)])
def test_prompt_attention_with_keys_in_two_parts(H, dim, rt, rank, dv, counts, window):
    """The tcgen05 kernel on packed prompts: windows shorter and longer than a tile, keys at both sides of every edge."""
    dev = _device("cuda")
    T, at, scale = sum(counts), H * (dim + rt), 0.5 / math.sqrt(dim + rt)
    ldz = -(-(at + rank + rt + H) // 8) * 8
    z, kv = rand(T, ldz, seed=1), rand(T, H * (dim + dv), seed=2)
    W = window or 10 ** 9
    z, kv = z.to(BF16), kv.to(BF16)
    first = [sum(counts[:i]) for i, c in enumerate(counts) for _ in range(c)]

    def key(j, h):
        return torch.cat((kv[j, h * dim:(h + 1) * dim], z[j, at + rank:at + rank + rt])).float()
    for i in range(0, T, 3):                              # the query looks at its window's edge, or just past it
        for h in range(H):
            j = i - W + 1 - (h % 2)
            if j < first[i]:
                j = first[i]
            k = key(j, h)
            z[i, h * (dim + rt):(h + 1) * (dim + rt)] = (10 / scale * k / k.norm() ** 2).to(BF16)
    start = torch.tensor(first, dtype=torch.int32, device=dev)
    gate = z[:, at + rank + rt:at + rank + rt + H]
    zd, kvd = z.to(dev)[:, :at + rank + rt + H], kv.to(dev)
    assert iops.latent_prefill_ok(zd, dim, rt, rank, dv)
    got = iops.attention_latent_prefill(zd, kvd, H, dim, rt, rank, dv, start, scale, window, zd[:, at + rank + rt:])
    k = torch.cat((kv[:, :H * dim].view(T, H, dim), z[:, at + rank:at + rank + rt].view(T, 1, rt).expand(-1, H, -1)), -1).double()
    v, q = kv[:, H * dim:].view(T, H, dv).double(), z[:, :at].view(T, H, dim + rt).double()
    want, a = [], 0
    for c in counts:
        want.append(plain.window_attention(q[a:a + c], k[a:a + c], v[a:a + c], scale, window))
        a += c
    close(got, torch.cat(want) * plain.sigmoid(gate.double())[..., None], 1.5e-2)
    plain_gate = iops.attention_latent_prefill(zd, kvd, H, dim, rt, rank, dv, start, scale, window)
    close(plain_gate, torch.cat(want), 1.5e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("window", [1, 9, 64, 65, 400])
def test_windowed_rows_and_prompts_of_plain_attention(device, window):
    """The window is an argument of the framework's other attention kernels too."""
    dev = _device(device)
    T, H, G, d = 150, 4, 2, 32
    q, k, v = rand(T, H, d, seed=1), rand(T, G, d, seed=2), rand(T, G, d, seed=3)
    rep = [h // 2 for h in range(H)]
    want = plain.window_attention(q.double(), k.double()[:, rep], v.double()[:, rep], 0.2, window)
    base = torch.zeros(T, dtype=torch.int32, device=dev)
    n = torch.arange(1, T + 1, dtype=torch.int32, device=dev)
    close(iops.attention_rows(q.to(dev), k.to(dev), v.to(dev), base, n, T, 0.2, window=window), want, 1e-5)
    if device == "cuda":
        qb, kb, vb = (x.to(BF16) for x in (q, k, v))
        wb = plain.window_attention(qb.double(), kb.double()[:, rep], vb.double()[:, rep], 0.2, window)
        close(iops.attention_prefill(qb.to(dev), kb.to(dev), vb.to(dev), base, 0.2, window=window), wb, 1.5e-2)


# ---- experts -------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,W,E,top,ff", [(1, 64, 6, 3, 64), (5, 52, 3, 3, 30), (200, 64, 6, 2, 96), (90, 128, 24, 5, 32),
                                          (70, 72, 4, 1, 160), (33, 64, 1, 1, 64), (300, 64, 3, 2, 40)])
def test_gated_experts_with_softmax_weights(device, dtype, n, W, E, top, ff):
    from easyllm_b200.models.hf_models.feedforward import SparseGLU
    dev = _device(device)
    h = rand(n, W, seed=1).to(dtype)
    w = {"m.router": rand(E, W, seed=2, scale=0.2), "m.router.b": rand(E, seed=3) * 2}
    for e in range(E):
        for i, (c, o, k) in enumerate((("gate", ff, W), ("up", ff, W), ("down", W, ff))):
            w[f"m.e{e}.{c}"] = rand(o, k, seed=10 + 3 * e + i, scale=k ** -0.5).to(dtype)
    w["m.router"] = w["m.router"].to(dtype)
    want = plain.moe(h.double(), {k: t.double() for k, t in w.items()}, "m", dict(router=dict(experts=E, top=top)))
    z = iops.linear_f32(h.to(dev), w["m.router"].to(dev))
    gu = torch.stack([SparseGLU.blocked(w[f"m.e{e}.gate"], w[f"m.e{e}.up"]) for e in range(E)])
    for e in range(E):
        assert all(torch.equal(a, w[f"m.e{e}.{c}"]) for a, c in zip(SparseGLU.split(gu[e]), ("gate", "up")))
    down = torch.stack([w[f"m.e{e}.down"] for e in range(E)])
    acc = rand(n, W, seed=5)
    got = iops.moe_glu_add_(acc.clone().to(dev), h.to(dev), z, w["m.router.b"].to(dev), top, gu.to(dev), SparseGLU.block_of(ff),
                            down.to(dev))
    d = (got.double().cpu() - acc.double() - want).abs().amax(-1) / want.abs().max()
    # in bf16 a close choice of experts may turn out the other way: a few rows may stand out
    assert float(d.max() if dtype == F32 else d.quantile(0.9)) < tol(dtype, 1e-5, 2e-2)


@pytest.mark.gpu
def test_router_weights_and_ties():
    _device("cuda")
    from easyllm_b200.ops import cuda_infer as ci
    z = torch.tensor([[1.0, 5.0, 5.0, -2.0, 0.0], [80.0, -80.0, 79.0, 0.0, 78.0]], device="cuda")
    b = torch.tensor([0.0, 0.0, 0.0, 10.0, 0.0], device="cuda")
    idx, w = ci.moe_route(z, 3, b, softmax=True)
    assert idx.tolist() == [[3, 1, 2], [0, 2, 4]]
    close(w[0], torch.softmax(torch.tensor([8.0, 5.0, 5.0]), -1), 1e-6)
    close(w[1], torch.softmax(torch.tensor([80.0, 79.0, 78.0]), -1), 1e-6)
