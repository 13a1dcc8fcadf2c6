"""Each mechanism of the hybrid decoder layers alone, against its plain statement: on the CPU and, marked gpu, the
kernels in fp32 and bf16, with sizes that hit and miss their vector and tensor-core paths."""
import math

import pytest
import torch

import plain_pafodra as plain
from easyllm_b200.ops import infer as iops

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
F32, BF16 = torch.float32, torch.bfloat16


def _device(name):
    if name == "cuda":
        if not torch.cuda.is_available():
            pytest.skip("no GPU")
        from easyllm_b200.ops import cuda
        cuda.lib()
    return torch.device(name)


def close(got, want, tol):
    d = (got.double().cpu() - want.double()).abs().max()
    assert d <= tol * max(1.0, float(want.abs().max())), float(d)


def rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def meta_of(counts, dev, slots=None, start=None):
    cu = [0]
    for c in counts:
        cu.append(cu[-1] + c)

    def t(x):
        return torch.tensor(x, dtype=torch.int32, device=dev)
    m = {"cu_seqlens": t(cu), "max_seqlen": max(counts)}
    if slots is not None:
        m.update(seq_slot=t(slots), seq_pos0=t(start))
    return m


# ---- matrix products ---------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,N,K", [(1, 5, 24), (1, 4096, 512), (3, 37, 50), (7, 264, 1032), (16, 1, 128), (70, 17, 64),
                                   (300, 520, 136), (33, 40, 20)])
def test_linear_forms(device, dtype, M, N, K):
    dev = _device(device)
    x, w, b = (t.to(dtype).to(dev) for t in (rand(M, K + 8, seed=1), rand(N, K, seed=2, scale=K ** -0.5), rand(N, seed=3)))
    want = x.double().cpu()[:, :K] @ w.double().cpu().t()
    tol = 2e-6 if dtype == F32 else 8e-3
    xs = x[:, :K]                                                  # a column slice of wider rows
    close(iops.linear(xs, w), want, tol)
    close(iops.linear(xs, w, b), want + b.double().cpu(), tol)
    close(iops.linear_f32(xs, w), want, 2e-6 if device == "cuda" or dtype == F32 else tol)
    close(iops.linear_act(xs, w, "tanh"), torch.tanh(want), tol)
    acc = rand(M, N, seed=4).to(dev)
    want_acc = rand(M, N, seed=4).double() + want
    assert iops.linear_add_(acc, xs.contiguous(), w) is acc
    close(acc, want_acc, 2e-6 if device == "cuda" or dtype == F32 else tol)
    ws = torch.stack([w, 2 * w, -w])
    xb = torch.stack([xs, xs + 1, xs])
    close(iops.linear_batch(xb, list(ws)), torch.stack([x_.double().cpu() @ w_.double().cpu().t() for x_, w_ in zip(xb, ws)]), tol)


def test_adjacent_parameters_alias_without_a_copy():
    ps = [torch.nn.Parameter(rand(n, 6, seed=n)) for n in (3, 5, 1)]
    before = torch.cat([p.detach() for p in ps])
    assert iops.fused_alias(ps) is None
    iops.make_adjacent_(ps)
    a = iops.fused_alias(ps)
    assert a is not None and torch.equal(a, before) and a.data_ptr() == ps[0].data_ptr()
    bs = [torch.nn.Parameter(rand(n, seed=n)) for n in (4, 2)]
    iops.make_adjacent_(bs)
    assert iops.fused_alias(bs).shape == (6,) and torch.equal(iops.fused(bs), torch.cat([b.detach() for b in bs]))


# ---- elementwise -------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [8, 30, 264])
def test_norm_embedding_and_activations(device, dtype, W):
    dev = _device(device)
    tol = 1e-6 if dtype == F32 else 8e-3
    x, w, b, add = rand(9, W, scale=3.0), rand(W, seed=1), rand(W, seed=2), rand(W, seed=3).to(dtype)
    xd = x.clone().to(dev)
    y = iops.dynamic_tanh(xd, torch.tensor(0.7).to(dev), w.to(dev), b.to(dev), dtype, add.to(dev))
    close(y, plain.dynamic_tanh(x.double(), torch.tensor(0.7).double(), w.double(), b.double()), tol)
    close(xd, x + add.float(), 1e-6)                       # the stream gains the bias after its norm was taken
    table = rand(11, W, seed=4).to(dtype)
    ids = torch.tensor([3, 10, 0, 3])
    close(iops.embed_scaled(ids.to(dev), table.to(dev), 5.25), table[ids].double() * 5.25, 1e-6)
    gu = rand(9, 2 * W, seed=5, scale=2.0).to(dtype)
    g, u = gu.double()[:, :W], gu.double()[:, W:]
    close(iops.glu(gu.to(dev), "gelu_tanh"), plain.gelu_tanh(g) * u, tol)
    close(iops.glu(gu.to(dev), "silu"), plain.silu(g) * u, tol)
    z = rand(9, 3, seed=6)
    close(iops.relu2_scaled(gu.to(dev), z.to(dev)[:, 1]), plain.sigmoid(z.double()[:, 1:2]) * gu.double().clamp(min=0) ** 2, tol)


# ---- attention -----------------------------------------------------------------------------------
def _rows(counts, dev):
    """kv_base / kv_len / row_start of packed fresh sequences."""
    base, length, at = [], [], 0
    for c in counts:
        base += [at] * c
        length += list(range(1, c + 1))
        at += c
    return [torch.tensor(x, dtype=torch.int32, device=dev) for x in (base, length)]


def _attention(q, k, v, counts, scale, sink, dev, prefill):
    base, length = _rows(counts, dev)
    q, k, v = q.to(dev), k.to(dev), v.to(dev)
    sink = None if sink is None else sink.to(dev)
    if prefill:
        assert iops.prefill_kernel_ok(q, v)
        return iops.attention_prefill(q, k, v, base, scale, sink)
    return iops.attention_rows(q, k, v, base, length, max(counts), scale, sink)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype,prefill", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (3, 1, 64, 8), (6, 6, 96, 72), (2, 1, 128, 128), (24, 2, 40, 104)])
def test_sink_attention(device, dtype, prefill, H, G, d, dv):
    dev = _device(device)
    if prefill and device == "cpu":
        pytest.skip("the prefill kernel needs a GPU")
    counts = [1, 45, 2]
    T = sum(counts)
    q, k, v = rand(T, H, d, seed=1).to(dtype), rand(T, G, d, seed=2).to(dtype), rand(T, G, dv, seed=3).to(dtype)
    for sink in (rand(H, seed=4) * 2, None):
        got = _attention(q, k, v, counts, 0.37, sink, dev, prefill)
        want, at = [], 0
        for c in counts:
            part = slice(at, at + c)
            want.append(plain.sink_attention(q[part].double(), k[part].double(), v[part].double(), 0.37,
                                             None if sink is None else sink.double()))
            at += c
        close(got, torch.cat(want), 2e-6 if dtype == F32 else 2e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,prefill", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("d,dv", [(64, 64), (96, 40), (128, 128)])
def test_far_keys_tile_edges_and_the_sink_stand_out(dtype, prefill, d, dv):
    """One key per query is the only one that scores: the first token, the neighbours of tile and range borders, the
    token itself.  Every other place reads almost nothing but the sink, so a wrong key, a key one place off, a lost
    first token or a sink that is left out (or counted twice) changes the value by its own size."""
    dev = _device("cuda")
    T, H, G = 1030, 4, 2
    targets = [0, 1, 63, 64, 127, 128, 129, 255, 256, 511, 512, 1023, 1024]
    gen = torch.Generator().manual_seed(0)
    code = torch.sign(torch.randn(T, d, generator=gen)) / math.sqrt(d)     # nearly orthogonal unit rows
    k = code.view(T, 1, d).repeat(1, G, 1)
    k[:, 1] = -k[:, 1]
    q = torch.zeros(T, H, d)
    v = torch.randn(T, G, dv, generator=gen)
    sink = torch.tensor([18.0, 20.0, 19.0, 21.0])
    hit = {}
    for i in range(T):
        seen = [t for t in targets if t <= i] + [i]
        hit[i] = [seen[(i + h) % len(seen)] for h in range(H)]
        for h in range(H):
            q[i, h] = k[hit[i][h], h // 2] * 20.0                          # score 20 at the target, about 20/sqrt(d) elsewhere
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    got = _attention(q, k, v, [T], 1.0, sink, dev, prefill).double().cpu()
    s = torch.einsum("qhd,khd->hqk", q.double(), k.double().repeat_interleave(2, 1))
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    p = torch.softmax(torch.cat((s, sink.double().view(H, 1, 1).expand(H, T, 1)), -1), -1)[..., :T]
    want = torch.einsum("hqk,khd->qhd", p, v.double().repeat_interleave(2, 1))
    assert max(float(p[h, i, hit[i][h]]) for i in (700, 1029) for h in range(H)) > 0.3
    close(got, want, 1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("device", DEVICES)
def test_cache_rows_of_several_slots(device):
    """Keys and values go to their slot and position; queries of different sequences read their own rows only, with the
    far part of the cache left full of another sequence's keys."""
    dev = _device(device)
    G, H, d, dv, cap = 2, 4, 24, 16, 300
    kc, vc = rand(3, cap, G, d, seed=1).to(dev) * 9, rand(3, cap, G, dv, seed=2).to(dev) * 9
    ks, vs = rand(290, G, d, seed=3), rand(290, G, dv, seed=4)
    sink = rand(H, seed=5)
    n2, n0 = 151, 130
    for slot, rows, pos in ((2, range(0, 151), range(0, 151)), (0, range(151, 281), range(0, 130))):
        m = {"kv_base": torch.full((len(rows),), slot * cap, dtype=torch.int32, device=dev),
             "kv_len": torch.tensor([p + 1 for p in pos], dtype=torch.int32, device=dev)}
        iops.kv_append(kc, vc, ks[list(rows)].to(dev), vs[list(rows)].to(dev), m)
    q = rand(3, H, d, seed=6)
    base = torch.tensor([2 * cap, 0, 2 * cap], dtype=torch.int32, device=dev)
    length = torch.tensor([n2, n0, 64], dtype=torch.int32, device=dev)
    got = iops.attention_rows(q.to(dev), kc.view(-1, G, d), vc.view(-1, G, dv), base, length, cap, 0.5, sink.to(dev))
    for t, (a, n) in enumerate(((0, n2), (151, n0), (0, 64))):
        want = plain.sink_attention(torch.cat((torch.zeros(n - 1, H, d), q[t:t + 1])).double(), ks[a:a + n].double(),
                                    vs[a:a + n].double(), 0.5, sink.double())[-1]
        close(got[t], want, 2e-6)


# ---- recurrences -----------------------------------------------------------------------------------
CUTS = [[40], [1] * 40, [16, 17, 7], [2, 3, 33, 1, 1]]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [20, 64, 1032])
def test_token_shift(device, dtype, W):
    dev = _device(device)
    h, mu = rand(40, W, seed=1).to(dtype), torch.rand(5, W, generator=torch.Generator().manual_seed(2))
    want = torch.stack([plain.token_shift(h.double(), m.double()) for m in mu])
    tol = 1e-6 if dtype == F32 else 2e-2
    close(iops.token_mix(h.to(dev), mu.to(dev), meta_of([40], dev), None), want, tol)
    for cuts in CUTS:
        tail, at, got = torch.full((3, W), 7.0, dtype=dtype, device=dev), 0, []
        for c in cuts:
            got.append(iops.token_mix(h[at:at + c].to(dev), mu.to(dev), meta_of([c], dev, [1], [at]), tail))
            at += c
        close(torch.cat(got, 1), want, tol)
        assert torch.equal(tail[1].cpu(), h[-1]) and bool((tail[[0, 2]] == 7).all())


def _scan_inputs(kind, H, G, d, dv, T, dtype):
    q, k, v = rand(T, G, d, seed=1), rand(T, G, d, seed=2, scale=d ** -0.5), rand(T, H, dv, seed=3)
    g = torch.exp(-torch.exp(rand(T, H, d, seed=4) - 3))
    if kind == "wkv":
        return q.to(dtype), k.to(dtype), v.to(dtype), g, rand(H, d, seed=5)
    return plain.unit(q) * d ** -0.5, plain.unit(k), v, g, torch.sigmoid(rand(T, H, seed=5))


def _scan(kind, ins, part, m, state, dev):
    a = [x[part].to(dev) for x in ins[:4]]
    if kind == "wkv":
        return iops.wkv_scan(*a, ins[4].to(dev), m, state)
    return iops.delta_scan(*a, ins[4][part].to(dev), m, state)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind,dtype", [("wkv", F32), ("wkv", BF16), ("delta", F32)])
@pytest.mark.parametrize("H,G,d,dv", [(2, 2, 32, 32), (4, 2, 20, 44), (2, 1, 128, 128), (1, 1, 200, 33), (3, 3, 64, 7)])
def test_scans(device, kind, dtype, H, G, d, dv):
    """A sequence in one piece, cut into steps, and beside others in a batch; the slot's old contents never show."""
    dev = _device(device)
    if kind == "wkv":
        G = H
    T = 40
    ins = _scan_inputs(kind, H, G, d, dv, T, dtype)
    which = [h // (H // G) for h in range(H)]
    qd, kd, vd, gd, ud = (x.double() for x in ins)
    want, S = (plain.wkv_recurrence(qd, kd, vd, gd, ud) if kind == "wkv"
               else plain.delta_recurrence(qd[:, which], kd[:, which], vd, gd, ud))
    tol = 4e-6
    close(_scan(kind, ins, slice(0, T), meta_of([T], dev), None, dev), want, tol)
    for cuts in CUTS:
        state = torch.full((3, H, dv, iops.padded_rows(d)), 5.0, device=dev)
        at, got = 0, []
        for c in cuts:
            got.append(_scan(kind, ins, slice(at, at + c), meta_of([c], dev, [2], [at]), state, dev))
            at += c
        close(torch.cat(got), want, tol)
        close(state[2][..., :d], S.transpose(1, 2), tol)
        assert bool((state[:2] == 5).all())
    # the same 40 tokens as three sequences of a batch, each in its own slot
    state = torch.full((4, H, dv, iops.padded_rows(d)), 5.0, device=dev)
    got = _scan(kind, ins, slice(0, T), meta_of([5, 1, 34], dev, [3, 0, 1], [0, 0, 0]), state, dev)
    at = 0
    for c, slot in ((5, 3), (1, 0), (34, 1)):
        p = slice(at, at + c)
        o, S = (plain.wkv_recurrence(qd[p], kd[p], vd[p], gd[p], ud) if kind == "wkv"
                else plain.delta_recurrence(qd[p][:, which], kd[p][:, which], vd[p], gd[p], ud[p]))
        close(got[p], o, tol)
        close(state[slot][..., :d], S.transpose(1, 2), tol)
        at += c


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind", ["wkv", "delta"])
def test_state_is_carried_far(device, kind):
    """A value written at the first token with a decay of almost one is read 3000 tokens later."""
    dev = _device(device)
    T, d = (3000 if device == "cuda" else 300), 16
    k, q, v = torch.zeros(T, 1, d), torch.zeros(T, 1, d), torch.zeros(T, 1, 8)
    k[0, 0, 3], q[-1, 0, 3], v[0] = 1.0, 1.0, torch.arange(1.0, 9.0)
    g = torch.full((T, 1, d), 0.9999)
    extra = torch.zeros(1, d) if kind == "wkv" else torch.ones(T, 1)
    o = _scan(kind, (q, k, v, g, extra), slice(0, T), meta_of([T], dev), None, dev)
    close(o[-1, 0], torch.arange(1.0, 9.0).double() * 0.9999 ** (T - 2 if kind == "wkv" else T - 1), 1e-4)
    assert bool((o[:-1] == 0).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,d,dv,taps", [(4, 2, 32, 48, 4), (3, 1, 10, 14, 2), (2, 2, 128, 64, 1), (2, 1, 24, 130, 17)])
def test_delta_inputs(device, dtype, H, G, d, dv, taps):
    """Short convolution, unit heads, decays and step sizes, over cuts that fall inside the convolution's reach."""
    dev = _device(device)
    T, C = 40, 2 * G * d + H * dv
    x, w = rand(T, C, seed=1).to(dtype), rand(C, taps, seed=2)
    a, A_log, dt, b = rand(T, H * d, seed=3, scale=3.0), rand(H, seed=4) - 2, rand(H * d, seed=5), rand(T, H + 3, seed=6)
    y = plain.silu(plain.short_conv(x.double(), w.double()))
    want = (plain.unit(y[:, :G * d].view(T, G, d)) * d ** -0.5, plain.unit(y[:, G * d:2 * G * d].view(T, G, d)),
            y[:, 2 * G * d:].view(T, H, dv),
            torch.exp(-torch.exp(A_log.double())[:, None] * plain.softplus(a.double() + dt.double()).view(T, H, d)),
            plain.sigmoid(b.double()[:, :H]))
    convs = [torch.nn.Parameter(p.to(dev)) for p in w.split([G * d, G * d, H * dv])]
    for cuts in CUTS:
        tail = torch.full((3, C, taps - 1), 4.0, dtype=dtype, device=dev)
        at, got = 0, []
        for c in cuts:
            p = slice(at, at + c)
            got.append(iops.delta_inputs(x[p].to(dev), convs, a[p].to(dev), A_log.to(dev), dt.to(dev), b.to(dev)[p, :H], H, G,
                                         d, dv, meta_of([c], dev, [1], [at]), tail))
            at += c
        for g, e in zip(zip(*got), want):
            close(torch.cat(list(g)), e, 3e-6)
        if taps > 1:
            assert torch.equal(tail[1].cpu(), x[T - taps + 1:].t())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,dv", [(3, 20), (1, 64), (4, 129)])
def test_head_norm_and_gate(device, dtype, H, dv):
    dev = _device(device)
    o, gate = rand(7, H, dv, seed=1, scale=0.02), rand(7, H * dv, seed=2).to(dtype)
    for w, act, fn in ((rand(H * dv, seed=3), "silu", plain.silu), (rand(dv, seed=4), "sigmoid", plain.sigmoid)):
        want = plain.over_rms(o.double(), 1e-4) * (w.double().view(-1, dv))
        want = want.reshape(7, -1) * fn(gate.double())
        close(iops.head_norm_gate(o.to(dev), w.to(dev), gate.to(dev), act, 1e-4, dtype), want, 2e-6 if dtype == F32 else 8e-3)


# ---- mixture of experts ------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,E,top,W,F", [(1, 8, 2, 64, 48), (5, 3, 3, 30, 21), (300, 6, 2, 128, 72), (200, 40, 1, 64, 264),
                                         (130, 1, 1, 64, 136)])
def test_mixture_of_experts(device, dtype, T, E, top, W, F):
    """Few tokens (row kernels) and many (grouped GEMM), experts with no token and with more than a tile of them."""
    dev = _device(device)
    h, z = rand(T, W, seed=1).to(dtype), rand(T, E, seed=2, scale=2.0)
    if E == 6:
        z[:, 4] = -9.0                                     # nobody's expert
        z[:200, 1] = 9.0                                   # more than one tile
    up, down = rand(E, F, W, seed=3, scale=W ** -0.5).to(dtype), rand(E, W, F, seed=4, scale=F ** -0.5).to(dtype)
    s = plain.sigmoid(z.double())
    want = rand(T, W, seed=5).double()
    acc = want.float().to(dev)
    for t in range(T):
        for e in z[t].topk(top).indices.tolist():
            want[t] += torch.clamp(up[e].double() @ (s[t, e] * h[t].double()), min=0) ** 2 @ down[e].double().t()
    iops.moe_relu2_add_(acc, h.to(dev), z.to(dev), top, up.to(dev), down.to(dev))
    close(acc, want, 3e-6 if dtype == F32 else 2e-2)
