"""Small random Megozen models for the tests: configs, weights under the checkpoint's tensor names."""
import math

import torch

from pafodra_models import save, tokens  # noqa: F401


def rot(dims, base=10000.0, **scaling):
    return dict(dims=dims, base=base, scaling=scaling) if scaling else dict(dims=dims, base=base)


def lat(heads, dim, rot_dim, vdim, rank, scale, window, r=None, **kw):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=scale, rot=r or rot(rot_dim))
    return dict(type="latent_attention", mixer=m if window is None else dict(m, mask=dict(size=window)), **kw)


def moe(experts, top, ff, shared=None):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    return m if shared is None else dict(m, shared=dict(ff=shared))


def config(vocab, width, layers, buckets, mul_prev, mul_cur, eps=1e-6):
    return dict(architecture="Megozen", vocab=vocab, width=width, layers=layers, norm=dict(eps=eps),
                embedding=dict(bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)))


YARN = dict(factor=8.0, original=64, fast=8.0, slow=0.5)
CONFIGS = {
    # sizes the TMA-fed kernels take: keys of one, two and three 64-column chunks; two layers on one set of weights; a
    # window of one tile and some, a short one, none
    "aligned": config(264, 128, [
        lat(4, 32, 16, 24, 48, 0.2, 19, rot(16, 500.0, **YARN), mlp=moe(6, 3, 64, 96)),
        lat(6, 64, 64, 64, 64, 0.11, 140, mlp=moe(5, 2, 96)),
        lat(20, 128, 64, 128, 96, 0.09, None, rot(64, 1000.0, **YARN), mlp=None),
        lat(4, 32, 16, 24, 48, 0.2, 19, rot(16, 500.0, **YARN), mlp=moe(6, 3, 64, 96), weights_of=0)], 101, 31, 7),
    # nothing is a multiple of 8; fewer rotated dimensions than the rotated part has; top = experts; a window of one token
    "odd": config(83, 52, [
        lat(3, 10, 6, 9, 13, 0.4, 11, rot(4, 300.0, factor=3.0, original=40, fast=4.0, slow=1.0), mlp=moe(3, 3, 30, 22)),
        lat(5, 7, 10, 18, 11, 0.3, 1, mlp=moe(4, 1, 21)),
        lat(3, 10, 6, 9, 13, 0.4, 11, rot(4, 300.0, factor=3.0, original=40, fast=4.0, slow=1.0), mlp=moe(3, 3, 30, 22),
            weights_of=0),
        lat(2, 5, 2, 4, 6, 0.8, None, mlp=None)], 17, 5, 3, eps=1e-3),
    # keys wider than the tensor-core prompt kernel takes, a latent row that is no multiple of 16, one expert, one head
    "wide": config(96, 64, [
        lat(33, 136, 40, 72, 144, 0.08, 50, mlp=moe(1, 1, 40, 8)), lat(1, 200, 24, 136, 72, 0.07, None, mlp=moe(9, 4, 32))],
        5, 2, 1),
}


def weights(cfg, seed=0, bf16=False):
    g = torch.Generator().manual_seed(seed)
    w = {}
    W, B = cfg["width"], cfg["embedding"]["bigram"]["buckets"]

    def mat(name, o, i, gain=1.0):
        w[name] = torch.randn(o, i, generator=g) * gain / math.sqrt(i)

    def vec(name, n, mean=0.0, std=1.0):
        w[name] = mean + std * torch.randn(n, generator=g)
    w["embed"], w["bigram"] = torch.randn(cfg["vocab"], W, generator=g), torch.randn(B + 1, W, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        n, m, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        vec(n + ".norm1", W, 1.0, 0.2)
        mat(n + ".mix.q", H * (d + r), W, 1.5), mat(n + ".mix.dkv", R + r, W, 1.5), vec(n + ".mix.dkv.norm", R, 1.0, 0.3)
        mat(n + ".mix.uk", H * d, R), mat(n + ".mix.uv", H * dv, R), mat(n + ".mix.g", H, W, 2.0), mat(n + ".mix.o", W, H * dv)
        if mlp:
            vec(n + ".norm2", W, 1.0, 0.2)
            mat(n + ".mlp.router", mlp["router"]["experts"], W, 2.0), vec(n + ".mlp.router.b", mlp["router"]["experts"])
            names = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            for e, ff in names + ([("shared", mlp["shared"]["ff"])] if "shared" in mlp else []):
                mat(f"{n}.mlp.{e}.gate", ff, W, 1.4), mat(f"{n}.mlp.{e}.up", ff, W), mat(f"{n}.mlp.{e}.down", W, ff, 1.4)
    vec("final.norm", W, 1.0, 0.2)
    mat("head", cfg["vocab"], W)
    return {n: t.to(torch.bfloat16) if bf16 else t for n, t in w.items()}
