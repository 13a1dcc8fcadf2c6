"""Serving throughput: prompts and decoding of a hybrid decoder beside the closest other model at equal size, and the
kernels of both one by one against their rooflines.

    python bench.py --serving [--serving-model pafodra|megozen] [--serving-sizes 2k,4k] [--serving-kernels]

Pafodra is measured beside a Llama, Megozen beside a Pafodra of attention layers with experts only.

Random weights; synthetic token ids.  Times are CUDA events on the launching stream, 3 warm-ups, medians.  The models
(gigabytes of weights) are far larger than L2; single kernels are timed with an L2 flush between iterations.  Prompts go
through ``CausalLM.step`` on fresh slots, decoding through the CUDA-graph step that ``generate`` replays.
"""
from __future__ import annotations

import gc
import json
import statistics

import torch

SIZES = {
    # width, attention heads, kv heads, ff, recurrent heads, experts, expert ff, layers, vocab
    "2k": dict(width=2048, heads=16, kv=8, ff=5632, rheads=16, experts=16, eff=1408, layers=10, vocab=32000),
    "4k": dict(width=4096, heads=32, kv=8, ff=11008, rheads=32, experts=16, eff=2752, layers=5, vocab=32000),
}


def pafodra_config(s):
    """Layers in the proportion attention : wkv : channel_delta = 2 : 2 : 1, half of the recurrent ones with experts."""
    d = 128
    att = {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": d, "vdim": d, "scale": d ** -0.5},
           "mlp": {"kind": "dense", "ff": s["ff"]}}
    moe = {"kind": "moe", "router": {"experts": s["experts"], "top": 2}, "expert": {"ff": s["eff"]}, "shared": {"ff": s["eff"]}}
    wkv = {"type": "wkv", "mixer": {"heads": s["width"] // 64, "dim": 64}}
    delta = {"type": "channel_delta", "mixer": {"heads": s["rheads"], "kv_heads": s["rheads"], "dim": d, "vdim": d, "conv": 4},
             "mlp": moe}
    period = [dict(wkv, mlp=moe), att, delta, att, dict(wkv, mlp={"kind": "dense", "ff": s["ff"]})]
    return {"architecture": "Pafodra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5},
            "embedding": {"scale": 4.0}, "layers": [period[i % 5] for i in range(s["layers"])]}


def pafodra_attention_config(s):
    """Attention layers with experts only: the closest relative of the Megozen below."""
    d = 128
    layer = {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": d, "vdim": d, "scale": d ** -0.5},
             "mlp": {"kind": "moe", "router": {"experts": s["experts"], "top": 2}, "expert": {"ff": s["eff"]},
                     "shared": {"ff": s["eff"]}}}
    return dict(pafodra_config(s), layers=[layer] * s["layers"])


# latent attention: heads of 128 unrotated + 64 rotated dimensions over a latent of 512, a window of 1024 tokens
LATENT = dict(dim=128, rot=64, vdim=128, rank=512, window=1024)


def megozen_config(s):
    m = LATENT
    rot = {"dims": m["rot"], "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    layer = {"type": "latent_attention",
             "mixer": {"heads": s["heads"], "dim": m["dim"], "rot_dim": m["rot"], "vdim": m["vdim"], "kv_rank": m["rank"],
                       "scale": (m["dim"] + m["rot"]) ** -0.5, "rot": rot, "mask": {"size": m["window"]}},
             "mlp": {"kind": "moe", "router": {"experts": s["experts"], "top": 2}, "expert": {"ff": s["eff"]},
                     "shared": {"ff": s["eff"]}}}
    return {"architecture": "Megozen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": s["vocab"] - 1, "mul_prev": 7919, "mul_cur": 104729}},
            "layers": [layer] * s["layers"]}


def build(which, s):
    from ..models.hf_models import CausalLM, HFArch, arch_from_hf_config
    configs = {"pafodra": pafodra_config, "pafodra attention": pafodra_attention_config, "megozen": megozen_config}
    arch = arch_from_hf_config(configs[which](s)) if which in configs else HFArch(
        family="llama", vocab_size=s["vocab"], hidden_size=s["width"], intermediate_size=s["ff"],
        num_hidden_layers=s["layers"], num_attention_heads=s["heads"], num_key_value_heads=s["kv"])
    torch.manual_seed(0)
    with torch.device("cuda"):
        model = CausalLM(arch, dtype=torch.bfloat16).eval()
    for n, p in model.named_parameters():        # decays spread as in a trained model, not all equal
        if n.endswith(".w0") or n.endswith(".A_log"):
            torch.nn.init.uniform_(p.data, -6.0, -1.0)
    return model


def _time(fn, iters):
    ts = []
    for i in range(iters + 3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        ts.append(a.elapsed_time(b))
    return statistics.median(ts[3:])


@torch.no_grad()
def bench_model(which, s, prefills, decodes, context, iters, sampler=None):
    from ..models.hf_models.state import DecodeGraph
    model = build(which, s)
    torch.cuda.synchronize()
    if sampler is not None:
        sampler.start()
    rows = []
    gen = torch.Generator().manual_seed(1)

    def prompt(n):
        return torch.randint(0, s["vocab"], (n,), generator=gen).cuda()
    for b, n in prefills:
        state = model.new_state(b, n)
        prompts = [prompt(n) for _ in range(b)]

        def once():
            slots = [state.open() for _ in range(b)]
            h, meta = model.step(state, slots, prompts)
            model.logits(h[meta["last_rows"].to(h.device, non_blocking=True)])
            for sl in slots:
                state.close(sl)
        ms = _time(once, iters)
        rows.append({"phase": "prefill", "batch": b, "tokens": n, "ms": round(ms, 3), "tokens_per_s": round(b * n / ms * 1e3)})
        del state
    for b in decodes:
        state = model.new_state(b, context + 4 * iters + 32)
        slots = [state.open() for _ in range(b)]
        for sl in slots:
            model.step(state, [sl], [prompt(context)])
        ids = prompt(b)
        model.logits(model.step(state, slots, ids)[0])
        graph = DecodeGraph(model, state, slots)
        ms = _time(lambda: graph.step(ids), iters)
        rows.append({"phase": "decode", "batch": b, "context": context, "ms": round(ms, 4), "tokens_per_s": round(b / ms * 1e3)})
        del state, graph
    n_params = sum(p.numel() for p in model.parameters())
    del model
    gc.collect()
    torch.cuda.empty_cache()
    return {"model": which, "parameters": n_params, "rows": rows}


def kernel_cases(s, T, B, context):
    """(kernel, phase, launch, bytes, flop, fp32-pipe flop) of the two models' layers at this size: bytes and operations
    the op cannot avoid."""
    from .. import ops
    from ..ops import cuda as cu
    from ..ops import cuda_infer as ci
    W, H, G, F, R, E, EF, D = s["width"], s["heads"], s["kv"], s["ff"], s["rheads"], s["experts"], s["eff"], 128
    bf, dev = torch.bfloat16, "cuda"

    def r(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(dtype)

    def meta(n_seq, each):
        return {"cu_seqlens": torch.arange(0, n_seq * each + 1, each, dtype=torch.int32, device=dev),
                "seq_slot": torch.arange(n_seq, dtype=torch.int32, device=dev),
                "seq_pos0": torch.full((n_seq,), 7, dtype=torch.int32, device=dev), "max_seqlen": each}
    f32 = torch.float32
    for phase, n, m in (("prefill", T, meta(1, T)), ("prefill8", T, meta(8, T // 8)), ("decode", B, meta(B, 1))):
        ns = m["cu_seqlens"].numel() - 1
        x32, h = r(n, W, dtype=f32), r(n, W)
        w1, b1, r_w = r(W, dtype=f32), r(W, dtype=f32), r(W)
        al = torch.tensor(0.5, device=dev)
        if phase != "prefill8":
            yield "dynamic_tanh", phase, lambda: ci.dynamic_tanh(x32, al, w1, b1, bf), 6 * n * W, 0, 0
            yield "llama rmsnorm+add", phase, lambda: cu.rmsnorm_fwd(h, h, r_w, 1e-6), 8 * n * W, 0, 0
            gu = r(n, 2 * F)
            yield "glu gelu", phase, lambda: ci.glu(gu, "gelu_tanh"), 6 * n * F, 0, 0
            yield "llama swiglu", phase, lambda: cu.swiglu_fwd(gu), 6 * n * F, 0, 0
            wq, wo = r(3 * W, W, scale=0.02), r(W, W, scale=0.02)
            yield "linear qkv", phase, lambda: ci.linear(h, wq), 2 * (n * W * 4 + 3 * W * W), 2 * n * W * 3 * W, 0
            yield "linear o += fp32", phase, lambda: ci.linear_add_(x32, h, wo), 2 * (n * W + W * W) + 8 * n * W, 2 * n * W * W, 0
            yield "llama linear o", phase, lambda: cu.gemm(h, wo), 2 * (2 * n * W + W * W), 2 * n * W * W, 0
        else:
            wq = wo = None
        mu = r(5, W, dtype=f32)
        last = r(ns, W)
        yield "token_mix", phase, lambda: ci.token_mix(h, mu, m, last), 12 * n * W, 0, 0
        hw, dw = W // 64, 64
        q, k, v = (r(n, hw, dw) for _ in range(3))
        dec, u = torch.rand(n, hw, dw, device=dev), r(hw, dw, dtype=f32)
        st = r(ns, hw, dw, 64, dtype=f32)
        yield ("wkv_scan", phase, lambda: ci.wkv_scan(q, k, v, dec, u, m, st), n * W * (6 + 4 + 4) + 8 * ns * W * dw, 0,
               n * hw * dw * dw * 5)
        q2, k2, v2, g2 = (torch.nn.functional.normalize(r(n, R, D, dtype=f32), dim=-1) for _ in range(4))
        beta = torch.rand(n, R, device=dev)
        st2 = r(ns, R, D, D, dtype=f32)
        gg = torch.rand(n, R, D, device=dev)
        yield ("delta_scan", phase, lambda: ci.delta_scan(q2, k2, v2, gg, beta, m, st2), n * R * D * 20 + 8 * ns * R * D * D, 0,
               n * R * D * D * 7)
        qkv, taps = r(n, 3 * R * D), r(3 * R * D, 4, dtype=f32)
        a, Al, dt, bb = r(n, R * D, dtype=f32), r(R, dtype=f32), r(R * D, dtype=f32), r(n, R, dtype=f32)
        tail = r(ns, 3 * R * D, 3)
        yield ("delta_inputs", phase, lambda: ci.delta_inputs(qkv, taps, a, Al, dt, bb, R, R, D, D, m, tail),
               n * R * D * (6 + 12 + 8), 0, 0)
        if phase == "prefill8":
            continue
        o32, gate, wn = r(n, R, D, dtype=f32), r(n, R * D), r(D, dtype=f32)
        yield "head_norm_gate", phase, lambda: ci.head_norm_gate(o32, wn, gate, "sigmoid", 1e-5, bf), n * R * D * 8, 0, 0
        z = r(n, E, dtype=f32)
        up, down = r(E, EF, W, scale=0.02), r(E, W, EF, scale=0.02)
        hit = min(E, 2 * n)
        yield ("experts (all launches)", phase, lambda: ci.moe_relu2_add_(x32, h, z, 2, up, down),
               2 * 2 * hit * EF * W + 2 * n * W + 8 * n * W, 2 * 2 * n * 2 * EF * W, 0)
        sink = r(H, dtype=f32)
        if phase == "prefill":
            q3, k3, v3 = r(n, H, D), r(n, G, D), r(n, G, D)
            rs = torch.zeros(n, dtype=torch.int32, device=dev)
            fl = 2 * n * n * D * H
            yield "attention + sink", phase, lambda: ci.attention_prefill(q3, k3, v3, rs, 0.09, sink), 2 * n * D * (2 * H + 2 * G), fl, 0
            yield "llama attention", phase, lambda: cu.flash_attn_fwd(q3, k3, v3, rs, 0.09), 2 * n * D * (2 * H + 2 * G), fl, 0
            q4, k4, v4 = r(n, H, 96), r(n, G, 96), r(n, G, 96)
            yield ("attention + sink, heads of 96", phase, lambda: ci.attention_prefill(q4, k4, v4, rs, 0.1, sink),
                   2 * n * 96 * (2 * H + 2 * G), 2 * n * n * 96 * H, 0)
        else:
            kc, vc = r(B * context, G, D), r(B * context, G, D)
            q3 = r(B, H, D)
            base = torch.arange(0, B * context, context, dtype=torch.int32, device=dev)
            ln = torch.full((B,), context, dtype=torch.int32, device=dev)
            yield ("attention rows + sink", phase, lambda: ci.attention_rows(q3, kc, vc, base, ln, context, 0.09, sink),
                   4 * B * context * G * D, 0, 0)
    del ops


def megozen_cases(s, T, B, context):
    """As ``kernel_cases``: Megozen's kernels, each followed by the like one of the other decoders."""
    from ..models.hf_models.feedforward import SparseGLU
    from ..models.layers import YarnRotaryTables
    from ..ops import cuda as cu
    from ..ops import cuda_infer as ci
    W, H, G, E, EF, V = s["width"], s["heads"], s["kv"], s["experts"], s["eff"], s["vocab"]
    d, r, dv, R, win = (LATENT[k] for k in ("dim", "rot", "vdim", "rank", "window"))
    bf, f32, dev = torch.bfloat16, torch.float32, "cuda"
    at, D = H * (d + r), 128

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(dtype)
    cos, sin = YarnRotaryTables(r, 1e4).get(context, torch.device(dev))
    for phase, n in (("prefill", T), ("decode", B)):
        x32, h = rnd(n, W, dtype=f32), rnd(n, W)
        w1, w2, al = rnd(W, dtype=f32), rnd(W, dtype=f32), torch.tensor(0.5, device=dev)
        pos = torch.arange(n, device=dev, dtype=torch.int32) % context
        m = {"position_ids": pos, "kv_base": torch.zeros(n, dtype=torch.int32, device=dev) if phase == "prefill" else
             torch.arange(0, n * context, context, dtype=torch.int32, device=dev), "kv_len": pos + 1}
        start = torch.zeros(n, dtype=torch.int32, device=dev)
        ids, table, pairs = torch.randint(0, V, (n,), device=dev), rnd(V, W), rnd(V, W)
        yield "layer_norms (two)", phase, lambda: ci.layer_norms(x32, [w1, w2], 1e-6, bf), 8 * n * W, 0, 0
        yield "like: dynamic_tanh", phase, lambda: ci.dynamic_tanh(x32, al, w1, w2, bf), 6 * n * W, 0, 0
        yield "embed_pairs", phase, lambda: ci.embed_pairs(ids, table, pairs, 1.0, 7919, 104729, start), 8 * n * W, 0, 0
        yield "like: embed_scaled", phase, lambda: ci.embed_scaled(ids, table, 2.0), 6 * n * W, 0, 0
        N = at + R + r + H
        win_, wq = rnd(N, W, scale=0.02), rnd((H + 2 * G) * D, W, scale=0.02)
        yield "linear q|latent|gate", phase, lambda: ci.linear(h, win_), 2 * (n * W + N * W + n * N), 2 * n * N * W, 0
        yield ("like: linear qkv", phase, lambda: ci.linear(h, wq), 2 * (n * W + wq.numel() + n * (H + 2 * G) * D),
               2 * n * wq.numel(), 0)
        z = ci.linear(h, win_)
        cache, nw = rnd(max(n if phase == "decode" else 1, 1), context, R + r), rnd(R, dtype=f32)
        q = rnd(n, H, R + r)
        moved = n * (4 * H * r + 6 * (R + r))
        yield ("latent_inputs", phase, lambda: ci.latent_inputs(z, H, d, r, R, nw, 1e-6, cos, sin, m, cache,
                                                                q[..., R:] if phase == "decode" else None), moved, 0, 0)
        qkv = rnd(n, 3 * H * D)
        c2, s2 = YarnRotaryTables(D, 1e4).get(context, torch.device(dev))
        yield ("like: rope of q and k", phase, lambda: cu.rope_(qkv, c2, s2, pos, 2 * H, D), n * 2 * H * D * 4, 0, 0)
        gu = torch.stack([SparseGLU.blocked(rnd(EF, W, scale=0.02), rnd(EF, W, scale=0.02)) for _ in range(E)])
        down, up = rnd(E, W, EF, scale=0.02), rnd(E, EF, W, scale=0.02)
        zr, hit = rnd(n, E, dtype=f32), min(E, 2 * n)
        yield ("gated experts (all launches)", phase, lambda: ci.moe_glu_add_(x32, h, zr, None, 2, gu, 32, down),
               2 * 3 * hit * EF * W + 2 * n * W + 8 * n * W, 2 * 2 * n * 3 * EF * W, 0)
        yield ("like: experts (all launches)", phase, lambda: ci.moe_relu2_add_(x32, h, zr, 2, up, down),
               2 * 2 * hit * EF * W + 2 * n * W + 8 * n * W, 2 * 2 * n * 2 * EF * W, 0)
        sg, wo, o = rnd(n, 2 * EF), rnd(W, H * dv, scale=0.02), rnd(n, H * dv)
        yield "glu silu (shared expert)", phase, lambda: ci.glu(sg, "silu"), 6 * n * EF, 0, 0
        yield "like: glu gelu", phase, lambda: ci.glu(sg, "gelu_tanh"), 6 * n * EF, 0, 0
        yield ("linear o += fp32", phase, lambda: ci.linear_add_(x32, o, wo), 2 * (n * H * dv + wo.numel()) + 8 * n * W,
               2 * n * wo.numel(), 0)
        gate = z[:, at + R + r:]
        if phase == "prefill":
            wkv = rnd(H * (d + dv), R, scale=0.04)
            yield ("linear latent -> k|v", phase, lambda: ci.linear(z[:, at:at + R], wkv),
                   2 * (n * R + wkv.numel() + n * H * (d + dv)), 2 * n * wkv.numel(), 0)
            kv = ci.linear(z[:, at:at + R], wkv)
            for w, seen in ((win, n * win - win * (win - 1) / 2), (None, n * (n + 1) / 2)):
                yield (f"latent attention, {'window %d' % w if w else 'all keys'}", phase,
                       lambda: ci.attention_latent_prefill(z, kv, H, d, r, R, dv, start, 0.07, w, gate),
                       2 * n * (at + R + r + 2 * H * (d + dv)), 2 * seen * H * (d + r + dv), 0)
            q3, k3, v3, sink = rnd(n, H, D), rnd(n, G, D), rnd(n, G, D), rnd(H, dtype=f32)
            yield ("like: attention + sink", phase, lambda: ci.attention_prefill(q3, k3, v3, start, 0.09, sink),
                   2 * n * D * (2 * H + 2 * G), 2 * n * n * D * H, 0)
        else:
            ukt, uv = rnd(H, R, d, scale=0.1), rnd(H, dv, R, scale=0.04)
            qn = z[:, :at].unflatten(1, (H, -1))[..., :d]
            yield ("query into the latent (per head)", phase, lambda: ci.head_products(qn, ukt, q[..., :R]),
                   2 * (ukt.numel() + n * H * (d + R)), 2 * n * ukt.numel(), 0)
            out, lat = torch.empty(n, H, dv, dtype=bf, device=dev), rnd(n, H, R)
            yield ("latent -> value (per head)", phase, lambda: ci.head_products(lat, uv, out),
                   2 * (uv.numel() + n * H * (dv + R)), 2 * n * uv.numel(), 0)
            for b in (1, B, 64):
                rows = rnd(b * context, R + r)
                qb, gb = rnd(b, H, R + r), rnd(b, H)
                base = torch.arange(0, b * context, context, dtype=torch.int32, device=dev)
                ln = torch.full((b,), context, dtype=torch.int32, device=dev)
                for w in (None, win):
                    keys = min(context, w or context)
                    yield (f"latent attention, batch {b}, {keys} keys", phase,
                           lambda: ci.attention_latent(qb, rows, R, base, ln, context, 0.07, w, gb),
                           2 * b * keys * (R + r), 2 * b * H * keys * (2 * R + r), 0)
                kc, vc, q3 = rnd(b * context, G, D), rnd(b * context, G, D), rnd(b, H, D)
                yield (f"like: attention rows, batch {b}, {context} keys", phase,
                       lambda: ci.attention_rows(q3, kc, vc, base, ln, context, 0.09), 4 * b * context * G * D, 0, 0)
                short = torch.full((b,), win, dtype=torch.int32, device=dev)
                yield (f"like: attention rows, batch {b}, {win} keys", phase,
                       lambda: ci.attention_rows(q3, kc, vc, base, short, win, 0.09), 4 * b * win * G * D, 0, 0)


FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12        # fp32 pipe at the highest SM clock


@torch.no_grad()
def bench_kernels(s, T=4096, B=8, context=4096, cases=kernel_cases):
    from ..ops.bench_kernels import _PEAKS, timed
    rows = []
    for name, phase, fn, nbytes, flop, fp32 in cases(s, T, B, context):
        us = timed(fn) * 1e3
        bounds = {"hbm": nbytes / (_PEAKS["hbm_gbs"] * 1e3), "tensor": flop / (_PEAKS["bf16_tflops"] * 1e6),
                  "fp32": fp32 / (FP32_TFLOPS * 1e6)}
        by = max(bounds, key=bounds.get)
        rows.append({"kernel": name, "phase": phase, "us": round(us, 1), "bound": by, "roofline_us": round(bounds[by], 1),
                     "fraction": round(bounds[by] / us, 3)})
        print(json.dumps(rows[-1]), flush=True)
    return rows, _PEAKS["source"]


def main(sizes, kernels=True, iters=20, clocks=None, model="pafodra"):
    """One JSON line per size; ``clocks``: a sampler with start() / stop() run around each model's timings
    (not around its making)."""
    from ..ops import cuda as cu
    cu.lib()
    for name in sizes:
        s = SIZES[name]
        for which in ("pafodra", "llama") if model == "pafodra" else ("megozen", "pafodra attention"):
            sampler = clocks() if clocks is not None else None
            l0 = cu.LAUNCHES
            out = bench_model(which, s, [(1, 4096), (8, 512), (1, 512)], [1, 8, 64], 4096, iters, sampler)
            out.update(size=name, shape=s, launches=cu.LAUNCHES - l0)
            if clocks is not None:
                out["clocks"] = sampler.stop()
            print(json.dumps(out), flush=True)
        cu.check_err_flag()
        if kernels:
            rows, source = bench_kernels(s, cases=kernel_cases if model == "pafodra" else megozen_cases)
            print(json.dumps({"size": name, "peaks": source, "kernels": rows}), flush=True)
            cu.check_err_flag()
    return 0
