"""Small random Pafodra models for the tests: configs, weights under the checkpoint's tensor names, folders on disk."""
import json
import math
import os

import torch


def att(heads, kv, dim, vdim, scale, **kw):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale), **kw)


def wkv(heads, dim, **kw):
    return dict(type="wkv", mixer=dict(heads=heads, dim=dim), **kw)


def delta(heads, kv, dim, vdim, conv, **kw):
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv), **kw)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, shared=None):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    return m if shared is None else dict(m, shared=dict(ff=shared))


def config(vocab, width, layers, scale=1.0, eps=1e-5):
    return dict(architecture="Pafodra", vocab=vocab, width=width, layers=layers, norm=dict(eps=eps), embedding=dict(scale=scale))


CONFIGS = {
    # sizes the TMA-fed kernels take; grouped value heads in the delta rule; two layers on one set of weights
    "aligned": config(264, 128, [
        delta(4, 2, 32, 48, 4, mlp=dense(160)), att(6, 2, 64, 40, 0.2, mlp=moe(8, 2, 64, 96)),
        wkv(4, 32, mlp=moe(5, 3, 48)), delta(4, 2, 32, 48, 4, mlp=dense(160), weights_of=0),
        att(4, 4, 96, 128, 0.11, mlp=None), att(6, 2, 64, 40, 0.2, mlp=moe(8, 2, 64, 96), weights_of=1)], scale=3.5),
    # nothing is a multiple of 8, one key/value head, two taps, top = experts
    "odd": config(83, 52, [
        wkv(3, 20, mlp=moe(3, 3, 30, 22)), att(5, 1, 12, 18, 0.4, mlp=dense(37)), delta(6, 3, 10, 14, 2, mlp=None),
        wkv(3, 20, mlp=moe(3, 3, 30, 22), weights_of=0)], scale=0.7, eps=1e-3),
    # heads wider than the tensor-core attention takes, no convolution history, one expert
    "wide": config(96, 64, [
        att(2, 1, 136, 144, 0.1, mlp=moe(1, 1, 40)), delta(2, 2, 160, 72, 1, mlp=dense(64)), wkv(1, 136, mlp=None)]),
}


def weights(cfg, seed=0, bf16=False):
    g = torch.Generator().manual_seed(seed)
    w = {}
    W = cfg["width"]

    def mat(name, o, i, gain=1.0):
        w[name] = torch.randn(o, i, generator=g) * gain / math.sqrt(i)

    def vec(name, *shape, mean=0.0, std=1.0):
        w[name] = mean + std * torch.randn(*shape, generator=g)

    def norm(name):
        vec(name, W, mean=1.0, std=0.2)
        vec(name + ".b", W, std=0.2)
        w[name + ".alpha"] = torch.tensor(0.6)
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        n, m = f"l{i}", layer["mixer"]
        norm(n + ".norm1")
        H, d = m["heads"], m["dim"]
        if layer["type"] == "attention":
            mat(n + ".mix.q", H * d, W, 1.5), mat(n + ".mix.k", m["kv_heads"] * d, W, 1.5)
            mat(n + ".mix.v", m["kv_heads"] * m["vdim"], W), mat(n + ".mix.o", W, H * m["vdim"])
            vec(n + ".mix.sink", H, mean=1.0)
        elif layer["type"] == "wkv":
            for c in "rkvg":
                mat(f"{n}.mix.{c}", H * d, W)
            for c in "rkvgw":
                w[f"{n}.mix.mu.{c}"] = torch.rand(W, generator=g)
            mat(n + ".mix.w1", 6 + 2 * i, W), mat(n + ".mix.w2", H * d, 6 + 2 * i)
            vec(n + ".mix.w0", H * d, mean=-3.0), vec(n + ".mix.u", H, d), vec(n + ".mix.norm", H * d, mean=1.0, std=0.3)
            mat(n + ".mix.o", W, H * d)
        else:
            qk, vv = m["kv_heads"] * d, H * m["vdim"]
            for c, k in (("q", qk), ("k", qk), ("v", vv)):
                mat(f"{n}.mix.{c}", k, W)
                vec(f"{n}.mix.{c}.conv", k, m["conv"], std=0.6)
            mat(n + ".mix.b", H, W, 2.0), mat(n + ".mix.a1", 8 + i, W), mat(n + ".mix.a2", H * d, 8 + i)
            mat(n + ".mix.g1", 16 - i, W), mat(n + ".mix.g2", vv, 16 - i), mat(n + ".mix.o", W, vv)
            vec(n + ".mix.A_log", H, mean=-2.0), vec(n + ".mix.dt_bias", H * d), vec(n + ".mix.norm", m["vdim"], mean=1.0, std=0.3)
        mlp = layer["mlp"]
        if mlp and mlp["kind"] == "dense":
            for c, o, k in (("gate", mlp["ff"], W), ("up", mlp["ff"], W), ("down", W, mlp["ff"])):
                mat(f"{n}.mlp.{c}", o, k)
                vec(f"{n}.mlp.{c}.b", o, std=0.3)
        elif mlp:
            mat(n + ".mlp.router", mlp["router"]["experts"], W, 2.0)
            for e in range(mlp["router"]["experts"]):
                mat(f"{n}.mlp.e{e}.up", mlp["expert"]["ff"], W, 1.4), mat(f"{n}.mlp.e{e}.down", W, mlp["expert"]["ff"])
            if "shared" in mlp:
                mat(n + ".mlp.shared.up", mlp["shared"]["ff"], W), mat(n + ".mlp.shared.down", W, mlp["shared"]["ff"])
                mat(n + ".mlp.shared.sg", 1, W, 2.0)
    norm("final.norm")
    mat("head", cfg["vocab"], W)
    return {n: t.to(torch.bfloat16) if bf16 else t for n, t in w.items()}


def save(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({n: t.contiguous() for n, t in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
