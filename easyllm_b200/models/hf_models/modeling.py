"""HuggingFace-style causal LMs for the data-parallel runner: one decoder, many families.

The reference vendors ~14 kLoC of per-family remote code patched to call flash-attn
(llm/models/hf_models/{llama,internlm,internlm2,baichuan,baichuan2,qwen}/modeling_*.py,
utils/flash_utils.py:62-655).  Here every family is one ``CausalLM`` parameterised by an
``HFArch`` record (RoPE vs ALiBi, q/k/v/o biases, GQA, norm-head, NTK / log-n scaling) that runs
on this framework's kernels: fused RMSNorm, RoPE on the packed QKV rows, causal segment-aware
flash attention (``cu_seqlens`` packing; padding is expressed as extra segments), SwiGLU and
the fused LM-head cross-entropy.  Checkpoints keep each family's own tensor names on disk
(``from_pretrained`` / ``save_pretrained`` translate through ``ckpt.hf_import`` rules).

Module attribute names follow HF Llama (``model.layers[i].self_attn`` …) so tools that walk the
module tree (Dynamic Checkpoint's ``level_keys: layers``, LoRA target names) work unchanged.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import List, Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from ... import ops
from ...ops import infer as iops
from ...ops import reference as ref
from ..layers import RotaryTables, alibi_slopes
from .feedforward import DenseGLU, SparseGLU, SparseMoE
from .latent import LatentAttention
from .mixers import ChannelDelta, DynamicTanh, LayerNorm, TimeMix
from .state import DecodeGraph, DecodeState, KVRows


@dataclass
class LayerSpec:
    """One layer of a decoder whose layers differ: the mixer and its sizes, the feed-forward (None: no feed-forward),
    and ``weights_of``, the layer whose tensors it uses (with a cache or state of its own)."""
    type: str = "attention"               # attention | wkv | channel_delta | latent_attention
    mixer: dict = field(default_factory=dict)
    mlp: Optional[dict] = None
    weights_of: Optional[int] = None


@dataclass
class HFArch:
    family: str = "llama"                 # llama | internlm | internlm2 | baichuan | baichuan2 | baichuan2-13b | qwen
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: Optional[int] = None
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    rope_scaling_factor: float = 1.0
    rope_dynamic_ntk_max_pos: Optional[int] = None
    max_position_embeddings: int = 4096
    qkv_bias: bool = False
    o_bias: bool = False
    position: str = "rope"                # rope | alibi
    norm_head: bool = False               # Baichuan2: rows of lm_head are L2-normalised
    use_logn_attn: bool = False           # Qwen inference-time log-n scaling of queries
    use_cache_quantization: bool = False  # Qwen: keep the decode KV cache in uint8 (per-chunk scale / zero)
    seq_length: int = 2048                # Qwen: training length for log-n / NTK
    tie_word_embeddings: bool = False
    pad_token_id: Optional[int] = None
    bos_token_id: Optional[int] = 1
    eos_token_id: Optional[int] = 2
    # decoders whose layers differ: one spec per layer (None: num_hidden_layers equal attention + SwiGLU layers), run as
    # parallel blocks x + mixer(norm x) + ff(norm x) on an fp32 stream
    layers: Optional[List[LayerSpec]] = None
    norm_eps: float = 1e-5                # eps of the layer norms and of the mixers' own norms
    embedding_scale: float = 1.0
    block_norm: str = "dynamic_tanh"      # dynamic_tanh: one norm for mixer and ff | layer_norm: one for each
    expert_form: str = "relu2"            # relu2: two matrices, input weighting | glu: three, softmax weights
    bigram: Optional[dict] = None         # table of (previous token, token) pairs: buckets, mul_prev, mul_cur

    @property
    def kv_heads(self):
        return self.num_key_value_heads or self.num_attention_heads

    @property
    def head_dim(self):
        return self.hidden_size // self.num_attention_heads


def arch_from_hf_config(cfg: dict, family: Optional[str] = None) -> HFArch:
    """Translate a family's ``config.json`` into an HFArch."""
    mt = (family or cfg.get("model_type") or cfg.get("architecture") or "llama").lower()
    if mt == "pafodra":
        return _pafodra_arch(cfg)
    if mt == "megozen":
        return _megozen_arch(cfg)
    a = HFArch(family=mt)
    g = cfg.get
    if mt == "qwen":
        a.vocab_size, a.hidden_size = g("vocab_size"), g("hidden_size")
        a.intermediate_size = g("intermediate_size", 4 * a.hidden_size) // 2   # Qwen stores 2·ffn
        a.num_hidden_layers, a.num_attention_heads = g("num_hidden_layers"), g("num_attention_heads")
        a.rms_norm_eps = g("layer_norm_epsilon", 1e-6)
        a.rope_theta = g("rotary_emb_base", 10000.0)
        a.qkv_bias, a.use_logn_attn, a.seq_length = True, g("use_logn_attn", False), g("seq_length", 2048)
        a.use_cache_quantization = bool(g("use_cache_quantization", False))
        a.rope_dynamic_ntk_max_pos = a.seq_length if g("use_dynamic_ntk", False) else None
        a.max_position_embeddings = g("max_position_embeddings", 8192)
        return a
    a.vocab_size, a.hidden_size = g("vocab_size", 32000), g("hidden_size", 4096)
    a.intermediate_size = g("intermediate_size", 11008)
    a.num_hidden_layers, a.num_attention_heads = g("num_hidden_layers", 32), g("num_attention_heads", 32)
    a.num_key_value_heads = g("num_key_value_heads")
    a.rms_norm_eps = g("rms_norm_eps", 1e-6)
    a.rope_theta = g("rope_theta", 10000.0)
    a.max_position_embeddings = g("max_position_embeddings", g("model_max_length", 4096))
    sc = g("rope_scaling") or {}
    if sc.get("type") == "linear":
        a.rope_scaling_factor = float(sc.get("factor", 1.0))
    elif sc.get("type") == "dynamic":
        a.rope_scaling_factor, a.rope_dynamic_ntk_max_pos = float(sc.get("factor", 1.0)), a.max_position_embeddings
    a.tie_word_embeddings = g("tie_word_embeddings", False)
    a.pad_token_id, a.bos_token_id, a.eos_token_id = g("pad_token_id"), g("bos_token_id", 1), g("eos_token_id", 2)
    if mt in ("internlm",):
        a.qkv_bias = a.o_bias = g("bias", True)
    if mt == "internlm2":
        a.qkv_bias = a.o_bias = g("bias", False)
    if mt in ("llama",):
        a.qkv_bias = a.o_bias = g("attention_bias", False)
    if mt.startswith("baichuan2"):
        a.norm_head = True
    if mt == "baichuan2-13b" or (mt.startswith("baichuan") and a.num_hidden_layers >= 40):
        a.position, a.family = "alibi", "baichuan2-13b" if mt.startswith("baichuan2") else mt
    return a


_MIXER_SIZES = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale"), "wkv": ("heads", "dim"),
                "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
                "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot")}


def _layer_specs(cfg: dict, mixers, mlps) -> List[LayerSpec]:
    """The 'layers' entries of a ``config.json``, checked; ``mixers`` / ``mlps``: the kinds this family has."""
    layers = []
    for i, e in enumerate(cfg["layers"]):
        if e["type"] not in mixers:
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        missing = [k for k in _MIXER_SIZES[e["type"]] if k not in e["mixer"]]
        if missing:
            raise ValueError(f"layer {i} ({e['type']}): the config has no {missing}")
        kv = e["mixer"].get("kv_heads")
        if kv and e["mixer"]["heads"] % kv:
            raise ValueError(f"layer {i}: {e['mixer']['heads']} heads do not divide into {kv} key/value heads")
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] not in mlps:
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        w = e.get("weights_of")
        if w is not None and not 0 <= w < len(cfg["layers"]):
            raise ValueError(f"layer {i}: weights_of {w} is not a layer")
        layers.append(LayerSpec(e["type"], dict(e["mixer"]), None if mlp is None else dict(mlp), w))
    return layers


def _megozen_arch(cfg: dict) -> HFArch:
    """``config.json`` of a Megozen model: vocab, width, norm.eps, embedding.bigram and one entry per layer."""
    layers = _layer_specs(cfg, ("latent_attention",), ("moe",))
    for i, l in enumerate(layers):
        dims = l.mixer["rot"]["dims"]
        if dims % 2 or l.mixer["rot_dim"] % 2 or not 0 < dims <= l.mixer["rot_dim"]:
            raise ValueError(f"layer {i}: {dims} rotated dimensions of {l.mixer['rot_dim']}")
        window = (l.mixer.get("mask") or {}).get("size")
        if window is not None and window < 1:
            raise ValueError(f"layer {i}: a window of {window} tokens")
    return HFArch(family="megozen", vocab_size=cfg["vocab"], hidden_size=cfg["width"], layers=layers,
                  num_hidden_layers=len(layers), num_attention_heads=layers[0].mixer["heads"] if layers else 1,
                  num_key_value_heads=1, norm_eps=cfg["norm"]["eps"], block_norm="layer_norm", expert_form="glu",
                  bigram=(cfg.get("embedding") or {}).get("bigram"), position="none", bos_token_id=cfg.get("bos_token_id"),
                  eos_token_id=cfg.get("eos_token_id"), pad_token_id=cfg.get("pad_token_id"))


def _pafodra_arch(cfg: dict) -> HFArch:
    """``config.json`` of a Pafodra model: vocab, width, norm.eps, embedding.scale and one entry per layer."""
    layers = _layer_specs(cfg, ("attention", "wkv", "channel_delta"), ("dense", "moe"))
    att = next((l.mixer for l in layers if l.type == "attention"), {})
    return HFArch(family="pafodra", vocab_size=cfg["vocab"], hidden_size=cfg["width"], layers=layers,
                  num_hidden_layers=len(layers), num_attention_heads=att.get("heads", 1),
                  num_key_value_heads=att.get("kv_heads", 1), norm_eps=cfg["norm"]["eps"],
                  embedding_scale=cfg["embedding"]["scale"], position="none", bos_token_id=cfg.get("bos_token_id"),
                  eos_token_id=cfg.get("eos_token_id"), pad_token_id=cfg.get("pad_token_id"))


def weight_owner(layers, i):
    """The layer whose tensors layer ``i`` uses (``weights_of`` followed to its end)."""
    seen = set()
    while layers[i].weights_of is not None and layers[i].weights_of != i:
        if i in seen:
            raise ValueError("weights_of runs in a circle")
        seen.add(i)
        i = layers[i].weights_of
    return i


class RMSNorm(nn.Module):
    def __init__(self, dim, eps, dtype):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim, dtype=dtype))
        self.eps = eps

    def forward(self, x, residual=None):
        if residual is None:
            return ops.rmsnorm(x, self.weight, self.eps)
        return ops.add_rmsnorm(x, residual, self.weight, self.eps)


class Attention(nn.Module):
    """Causal attention: GQA, RoPE / ALiBi / no positions, value heads of another size than the keys', a given score
    scale, and a learned sink per head in the softmax denominator.  ``m``: sizes of this layer (None: the arch's)."""

    def __init__(self, a: HFArch, dtype, m: Optional[dict] = None):
        super().__init__()
        self.a = a
        m = m or {"heads": a.num_attention_heads, "kv_heads": a.kv_heads, "dim": a.head_dim, "vdim": a.head_dim}
        d, dv, hq, hk = m["dim"], m["vdim"], m["heads"], m["kv_heads"]
        self.d, self.dv, self.hq, self.hk = d, dv, hq, hk
        self.scale = float(m.get("scale", 1.0 / math.sqrt(d)))
        self.q_proj = nn.Linear(a.hidden_size, hq * d, bias=a.qkv_bias, dtype=dtype)
        self.k_proj = nn.Linear(a.hidden_size, hk * d, bias=a.qkv_bias, dtype=dtype)
        self.v_proj = nn.Linear(a.hidden_size, hk * dv, bias=a.qkv_bias, dtype=dtype)
        self.o_proj = nn.Linear(hq * dv, a.hidden_size, bias=a.o_bias, dtype=dtype)
        self.sink = nn.Parameter(torch.zeros(hq)) if m.get("sink") else None
        self.rotary = RotaryTables(d, a.rope_theta, a.rope_scaling_factor, a.rope_dynamic_ntk_max_pos) \
            if a.position == "rope" else None
        self.slopes = torch.tensor(alibi_slopes(hq), dtype=torch.float32) if a.position == "alibi" else None

    def fused_groups(self):
        ps = (self.q_proj, self.k_proj, self.v_proj)
        return [[p.weight for p in ps]] + ([[p.bias for p in ps]] if self.a.qkv_bias else [])

    def new_state(self, slots, capacity, device, dtype):
        if self.a.use_cache_quantization:
            from .kv_quant import QuantizedKV
            return {"kq": QuantizedKV(slots, capacity, self.hk, self.d, device, dtype),
                    "vq": QuantizedKV(slots, capacity, self.hk, self.dv, device, dtype), "len": 0}
        return KVRows(slots, capacity, self.hk, self.d, self.dv, device, dtype)

    def _split(self, qkv):
        T, nq, nk = qkv.shape[0], self.hq * self.d, self.hk * self.d
        return (qkv[:, :nq].view(T, self.hq, self.d), qkv[:, nq:nq + nk].view(T, self.hk, self.d),
                qkv[:, nq + nk:].view(T, self.hk, self.dv))

    def _attend(self, q, k, v, meta, cache):
        """Serving attention: prompts that start here on the prefill kernel, everything else over the cached rows.
        ``cache``: the layer's ``KVRows``, or None for packed sequences that keep nothing."""
        T = q.shape[0]
        sl = self.slopes.to(q.device) if self.slopes is not None else None
        sink = self.sink.detach() if self.sink is not None else None
        if cache is not None:
            iops.kv_append(cache.k, cache.v, k, v, meta)
        fresh = cache is None or (meta["fresh"] and not meta["one_token"])
        if fresh and iops.prefill_kernel_ok(q, v):
            row_start = meta["row_start"]
            if row_start is None:
                row_start = ops.cuda.row_start_of(meta["cu_seqlens"], T, q.device)
            o = iops.attention_prefill(q, k, v, row_start, self.scale, sink, sl)
        elif cache is not None:
            o = iops.attention_rows(q, cache.k.view(-1, self.hk, self.d), cache.v.view(-1, self.hk, self.dv),
                                    meta["kv_base"], meta["kv_len"], meta.get("kv_bound", meta["max_position"]),
                                    self.scale, sink, sl)
        else:
            cu = meta["cu_seqlens"].long()
            start = torch.repeat_interleave(cu[:-1], cu[1:] - cu[:-1], output_size=T)
            n = torch.arange(T, device=q.device) - start + 1
            o = iops.attention_rows(q, k, v, start.int(), n.int(), meta["max_seqlen"], self.scale, sink, sl)
        return o.reshape(T, self.hq * self.dv)

    def forward(self, x, meta, cache=None, residual=None):
        """``residual``: fp32 stream the output projection is accumulated into (parallel blocks, inference only)."""
        if residual is not None:
            qkv = iops.linear_cat(x, [self.q_proj.weight, self.k_proj.weight, self.v_proj.weight],
                                  [self.q_proj.bias, self.k_proj.bias, self.v_proj.bias] if self.a.qkv_bias else None)
            o = self._attend(*self._split(qkv), meta, cache)
            return iops.linear_add_(residual, o, self.o_proj.weight)
        a = self.a
        d, hq, hk = self.d, self.hq, self.hk
        T = x.shape[0]
        qkv = ops.linear_parts(x, (self.q_proj.weight, self.k_proj.weight, self.v_proj.weight),
                               (self.q_proj.bias, self.k_proj.bias, self.v_proj.bias) if a.qkv_bias else None)
        pos = meta["position_ids"]
        rope = None
        if self.rotary is not None:
            cos, sin = self.rotary.get(int(meta["max_position"]), x.device)
            rope = (cos, sin, pos)
        if cache is None and not (a.use_logn_attn and not self.training):
            # training / full-sequence path: RoPE + attention on the packed projection, one packed gradient back
            sl = self.slopes.to(x.device) if self.slopes is not None else None
            o = ops.flash_attention_packed(qkv, hq, hk, d, meta["cu_seqlens"], meta["max_seqlen"], alibi_slopes=sl,
                                           rope=rope, row_start=meta.get("row_start"))
            return ops.linear(o, self.o_proj.weight, self.o_proj.bias)
        if rope is not None:
            qkv = ops.rope_packed(qkv, cos, sin, pos, hq, hk, d)
        q, k, v = self._split(qkv)
        if a.use_logn_attn and not self.training:
            logn = torch.clamp(torch.log(pos.float() + 1) / math.log(a.seq_length), min=1.0)
            q = (q.float() * logn.view(T, 1, 1)).to(q.dtype)
        if isinstance(cache, KVRows):
            o = self._attend(q, k, v, meta, cache)
        elif cache is not None:               # dense batch of equal length in a dict: 8-bit cache, draft trees, prefixes
            B = meta["batch"]
            S = T // B
            p0 = cache["len"]
            cache_ref = cache
            if "kq" in cache:                 # 8-bit cache: quantise the new chunk, attend over the dequantised prefix
                cache["kq"].append(p0, k.reshape(B, S, hk, d))
                cache["vq"].append(p0, v.reshape(B, S, hk, d))
                cache = dict(cache, k=cache["kq"].read(p0 + S), v=cache["vq"].read(p0 + S))
                cache_ref["len"] = p0 + S
            else:
                cache["k"][:, p0:p0 + S] = k.reshape(B, S, hk, d)
                cache["v"][:, p0:p0 + S] = v.reshape(B, S, hk, d)
                cache["len"] = p0 + S
            if meta.get("tree_mask") is not None:
                o = _tree_cached(q.reshape(B, S, hq, d), cache["k"][:, :p0 + S], cache["v"][:, :p0 + S], p0,
                                 meta["tree_mask"])
            elif self.slopes is not None:
                o = _alibi_cached(q.reshape(B, S, hq, d), cache["k"][:, :p0 + S], cache["v"][:, :p0 + S], p0,
                                  self.slopes.to(x.device))
            else:
                o = ref.attention_kvcache(q.reshape(B, S, hq, d), cache["k"][:, :p0 + S], cache["v"][:, :p0 + S], p0)
            o = o.reshape(T, hq * d)
        else:
            sl = self.slopes.to(x.device) if self.slopes is not None else None
            o = ops.flash_attention(q, k, v, meta["cu_seqlens"], meta["max_seqlen"], True, alibi_slopes=sl)
            o = o.reshape(T, hq * d)
        return ops.linear(o, self.o_proj.weight, self.o_proj.bias)


def _tree_cached(q, kc, vc, p0, tree_mask):
    """Speculative-tree attention: every draft node sees the whole prefix cache and its ancestors."""
    B, Sq, H, D = q.shape
    rep = H // kc.shape[2]
    s = torch.einsum("bqhd,bkhd->bhqk", q.float(), kc.float().repeat_interleave(rep, 2)) / math.sqrt(D)
    full = torch.ones(Sq, p0 + Sq, dtype=torch.bool, device=q.device)
    full[:, p0:] = tree_mask
    s = s.masked_fill(~full.view(1, 1, Sq, p0 + Sq), float("-inf"))
    return torch.einsum("bhqk,bkhd->bqhd", torch.softmax(s, -1), vc.float().repeat_interleave(rep, 2)).to(q.dtype)


def _alibi_cached(q, kc, vc, p0, slopes):
    B, Sq, H, D = q.shape
    Sk = kc.shape[1]
    rep = H // kc.shape[2]
    s = torch.einsum("bqhd,bkhd->bhqk", q.float(), kc.float().repeat_interleave(rep, 2)) / math.sqrt(D)
    qi = torch.arange(Sq, device=q.device).view(Sq, 1) + p0
    kj = torch.arange(Sk, device=q.device).view(1, Sk)
    s = s + slopes.view(1, H, 1, 1) * (kj - qi).view(1, 1, Sq, Sk)
    s = s.masked_fill((kj > qi).view(1, 1, Sq, Sk), float("-inf"))
    return torch.einsum("bhqk,bkhd->bqhd", torch.softmax(s, -1), vc.float().repeat_interleave(rep, 2)).to(q.dtype)


class MLP(nn.Module):
    def __init__(self, a: HFArch, dtype):
        super().__init__()
        self.gate_proj = nn.Linear(a.hidden_size, a.intermediate_size, bias=False, dtype=dtype)
        self.up_proj = nn.Linear(a.hidden_size, a.intermediate_size, bias=False, dtype=dtype)
        self.down_proj = nn.Linear(a.intermediate_size, a.hidden_size, bias=False, dtype=dtype)

    def forward(self, x):
        gu = ops.linear_parts(x, (self.gate_proj.weight, self.up_proj.weight))
        return ops.linear(ops.glu(gu, "silu"), self.down_proj.weight)


class DecoderLayer(nn.Module):
    def __init__(self, a: HFArch, dtype):
        super().__init__()
        self.self_attn = Attention(a, dtype)
        self.mlp = MLP(a, dtype)
        self.input_layernorm = RMSNorm(a.hidden_size, a.rms_norm_eps, dtype)
        self.post_attention_layernorm = RMSNorm(a.hidden_size, a.rms_norm_eps, dtype)

    def new_state(self, *a):
        return self.self_attn.new_state(*a)

    def forward(self, delta, residual, meta, cache=None):
        if residual is None:
            h = delta
            n1 = self.input_layernorm(h)
        else:
            n1, h = self.input_layernorm(delta, residual)
        n2, h = self.post_attention_layernorm(self.self_attn(n1, meta, cache), h)
        return self.mlp(n2), h


def _block_norm(a: HFArch, dtype):
    return DynamicTanh(a.hidden_size, dtype) if a.block_norm == "dynamic_tanh" else LayerNorm(a.hidden_size, a.norm_eps, dtype)


class ParallelLayer(nn.Module):
    """``x + mixer(norm x) + ff(norm x)``: both sublayers accumulate into the fp32 stream ``x``.  They share one norm, or
    (``block_norm: layer_norm``) have one each, taken from the same ``x`` in one pass."""

    def __init__(self, a: HFArch, spec: LayerSpec, dtype):
        super().__init__()
        m = spec.mixer
        self.input_layernorm = _block_norm(a, dtype)
        self.mlp_layernorm = _block_norm(a, dtype) if a.block_norm == "layer_norm" and spec.mlp is not None else None
        if spec.type == "attention":
            self.mixer = Attention(a, dtype, dict(m, sink=True))
        else:
            self.mixer = {"wkv": TimeMix, "channel_delta": ChannelDelta,
                          "latent_attention": LatentAttention}[spec.type](a.hidden_size, m, a.norm_eps, dtype)
        self.mlp = None
        if spec.mlp is not None:
            self.mlp = DenseGLU(a.hidden_size, spec.mlp["ff"], "gelu_tanh", dtype) if spec.mlp["kind"] == "dense" \
                else (SparseGLU if a.expert_form == "glu" else SparseMoE)(a.hidden_size, spec.mlp, dtype)

    def new_state(self, *a):
        return self.mixer.new_state(*a)

    def forward(self, x, _residual, meta, cache=None):
        if self.mlp_layernorm is not None:
            h, hf = self.input_layernorm(x, self.mlp_layernorm)
        else:
            h = hf = self.input_layernorm(x, self.mlp.out_bias if self.mlp is not None else None)
        self.mixer(h, meta, cache, x)
        if self.mlp is not None:
            self.mlp(hf, x)
        return x, None


class Decoder(nn.Module):
    def __init__(self, a: HFArch, dtype):
        super().__init__()
        self.embed_tokens = nn.Embedding(a.vocab_size, a.hidden_size, dtype=dtype)
        self.embedding_scale, self.hybrid, self.bigram = a.embedding_scale, a.layers is not None, a.bigram
        self.keeps_tokens = a.bigram is not None          # the state holds token ids: the embedding looks one back
        if self.bigram is not None:
            self.embed_pairs = nn.Embedding(self.bigram["buckets"] + 1, a.hidden_size, dtype=dtype)
        if self.hybrid:
            own = {i: ParallelLayer(a, a.layers[i], dtype) for i in {weight_owner(a.layers, i) for i in range(len(a.layers))}}
            # a layer with the weights of another one is the same module at two places, with a state at each
            self.layers = nn.ModuleList(own[weight_owner(a.layers, i)] for i in range(len(a.layers)))
            self.norm = _block_norm(a, dtype)
        else:
            self.layers = nn.ModuleList(DecoderLayer(a, dtype) for _ in range(a.num_hidden_layers))
            self.norm = RMSNorm(a.hidden_size, a.rms_norm_eps, dtype)

    def embed(self, ids, meta=None, tokens=None):
        """The residual stream the layers start from.  ``meta`` and ``tokens`` (what the state keeps of earlier steps, or
        None) matter where the embedding looks at the previous token."""
        if self.bigram is not None:
            return iops.embed_pairs(ids.reshape(-1), self.embed_tokens.weight, self.embed_pairs.weight, self.embedding_scale,
                                    self.bigram["mul_prev"], self.bigram["mul_cur"], meta,
                                    tokens.ids if tokens is not None else None)
        if self.hybrid:
            return iops.embed_scaled(ids.reshape(-1), self.embed_tokens.weight, self.embedding_scale)
        return self.embed_tokens(ids.reshape(-1))


def build_meta(input_ids, attention_mask=None, position_ids=None, cu_seqlens=None, device=None):
    """Token-major metadata.  Padding becomes its own segments so real tokens never see it.
    Everything is computed where ``input_ids`` lives and then moved to ``device``: with a batch still on the host
    (as a loader delivers it) the scalars below cost no device→host synchronisation."""
    b, s = input_ids.shape
    dev = input_ids.device
    out_dev = torch.device(device) if device is not None else dev
    if cu_seqlens is not None:
        cu = torch.unique_consecutive(cu_seqlens.reshape(-1).to(torch.int32))
        if int(cu[-1]) < b * s:
            cu = torch.cat((cu, cu.new_tensor([b * s])))
    else:
        bounds = set(range(0, (b + 1) * s, s))
        if attention_mask is not None and not bool(attention_mask.all()):
            m = attention_mask.bool()
            for i in range(b):
                edges = torch.nonzero(m[i, 1:] != m[i, :-1]).flatten() + 1
                bounds.update(i * s + int(e) for e in edges)
        cu = torch.tensor(sorted(bounds), dtype=torch.int32, device=dev)
    if position_ids is None:
        if attention_mask is not None and not bool(attention_mask.all()):
            position_ids = (attention_mask.long().cumsum(-1) - 1).clamp(min=0)
        else:
            position_ids = torch.arange(s, device=dev).unsqueeze(0).expand(b, s)
    pos = position_ids.reshape(-1).to(torch.int32)
    meta = {"max_seqlen": int((cu[1:] - cu[:-1]).max()), "batch": b, "max_position": max(s, int(pos.max()) + 1)}
    row_start = None
    if out_dev.type == "cuda":
        from ...ops import cuda as cu_ops
        if cu_ops.available():
            row_start = cu_ops.row_start_of(cu, b * s, out_dev)   # once per batch, not once per layer
    meta.update(position_ids=pos.to(out_dev, non_blocking=True), cu_seqlens=cu.to(out_dev, non_blocking=True),
                row_start=row_start)
    return meta


def _penalise(logits, toks, seen, values):
    """``logits[r, toks[r, c]] = values[r, c]`` where ``seen`` (padding columns must not touch their id's logit)."""
    r, c = torch.nonzero(seen, as_tuple=True)
    logits = logits.clone()
    logits[r, toks[r, c]] = values[r, c]
    return logits


class CausalLM(nn.Module):
    def __init__(self, arch: HFArch, dtype=torch.float32):
        super().__init__()
        self.arch = arch
        self.config = arch
        self.model = Decoder(arch, dtype)
        self.lm_head = nn.Linear(arch.hidden_size, arch.vocab_size, bias=False, dtype=dtype)
        self.gradient_checkpointing = False
        self.apply(self._init)

    @staticmethod
    def _init(m):
        if isinstance(m, (nn.Linear, nn.Embedding)):
            nn.init.normal_(m.weight, 0.0, 0.02)
            if getattr(m, "bias", None) is not None:
                nn.init.zeros_(m.bias)

    def gradient_checkpointing_enable(self, **_):
        self.gradient_checkpointing = True

    def gradient_checkpointing_disable(self):
        self.gradient_checkpointing = False

    def get_input_embeddings(self):
        return self.model.embed_tokens

    def head_weight(self):
        w = self.lm_head.weight
        return F.normalize(w.float(), dim=-1).to(w.dtype) if self.arch.norm_head else w

    def prepare_positions(self, length, device):
        """Position tables for sequences of up to ``length`` tokens, made now rather than in a step."""
        for m in self.modules():
            if getattr(m, "rotary", None) is not None:
                m.rotary.get(length, device)

    def hidden_states(self, input_ids, meta, caches=None, inputs_embeds=None, tokens=None):
        if inputs_embeds is not None and self.model.keeps_tokens:
            raise NotImplementedError(f"{self.arch.family}: the embedding depends on token pairs, it takes ids only")
        x = inputs_embeds if inputs_embeds is not None else self.model.embed(input_ids, meta, tokens)
        x = x.reshape(-1, x.shape[-1])
        if self.model.hybrid:
            iops.no_grad_check(x, self.lm_head.weight)
            x = x.float() if inputs_embeds is None else x.to(torch.float32, copy=True)     # the layers write into it
        delta, residual = x, None
        for i, layer in enumerate(self.model.layers):
            cache = caches[i] if caches is not None else None
            if self.gradient_checkpointing and self.training and cache is None:
                from torch.utils.checkpoint import checkpoint
                delta, residual = checkpoint(lambda d, r, _l=layer: _l(d, r, meta), delta, residual, use_reentrant=False)
            else:
                delta, residual = layer(delta, residual, meta, cache)
        if residual is None:
            return self.model.norm(delta)
        return self.model.norm(delta, residual)[0]

    def forward(self, input_ids=None, attention_mask=None, labels=None, position_ids=None, cu_seqlens=None,
                inputs_embeds=None, return_dict=True, **_):
        if self.model.hybrid and labels is not None:
            raise NotImplementedError(f"{self.arch.family}: the hybrid decoder layers are inference-only (no loss)")
        b, s = input_ids.shape
        dev = self.lm_head.weight.device
        # a batch handed over on the host is parsed there and copied (no read-back from the GPU per micro-batch)
        meta = build_meta(input_ids, attention_mask, position_ids, cu_seqlens, device=dev)
        input_ids = input_ids.to(dev, non_blocking=True)
        if labels is not None:
            labels = labels.to(dev, non_blocking=True)
        if self.model.hybrid:
            with torch.no_grad():
                h = self.hidden_states(input_ids, meta, inputs_embeds=inputs_embeds)
                return {"logits": self.logits(h).view(b, s, -1)}
        h = self.hidden_states(input_ids, meta, inputs_embeds=inputs_embeds)
        out = {}
        if labels is not None:
            # HF convention: the model shifts — position t predicts labels[t + 1]
            shift = torch.full_like(labels, -100)
            shift[:, :-1] = labels[:, 1:]
            flat = shift.reshape(-1)
            valid = flat != -100
            tok = ops.lm_head_cross_entropy(h, self.head_weight(), flat.masked_fill(~valid, 0))
            out["loss"] = (tok * valid).sum() / valid.sum().clamp(min=1)
            with torch.no_grad():
                out["num_tokens"] = valid.sum()
        else:
            out["logits"] = ops.linear(h, self.head_weight()).view(b, s, -1)
        return out

    # ---- generation -----------------------------------------------------------------------------
    def fuse_weights(self):
        """Put the projections that are applied together next to each other in memory (once; a no-op afterwards)."""
        for m in self.modules():
            for group in getattr(m, "fused_groups", list)():
                iops.make_adjacent_(group)

    def new_state(self, slots, capacity):
        """The cache / state manager of up to ``slots`` sequences of ``capacity`` tokens (it grows when that is not
        enough)."""
        self.fuse_weights()
        return DecodeState(self, slots, capacity)

    @torch.no_grad()
    def step(self, state, slots, tokens, inputs_embeds=None):
        """Run the next tokens of the sequences in ``slots`` as one batch, from what ``state`` holds of them.
        ``tokens``: list of 1-D id tensors / lists (unequal lengths are packed, not padded), or one id per sequence as
        a device tensor ``[n]``.  Returns the normed hidden rows of all tokens and the step's meta (``last_rows``: the
        row of every sequence's last token)."""
        dev = self.lm_head.weight.device
        if torch.is_tensor(tokens):
            counts, ids = [1] * len(slots), tokens.reshape(-1).to(dev)
        else:
            parts = [torch.as_tensor(t, dtype=torch.long).reshape(-1) for t in tokens]
            counts, ids = [p.numel() for p in parts], torch.cat(parts).to(dev, non_blocking=True)
        meta = state.step_meta(slots, counts)
        return self.hidden_states(ids, meta, state.layers, inputs_embeds=inputs_embeds, tokens=state.tokens), meta

    @torch.no_grad()
    def logits(self, h):
        """fp32 logits of hidden rows."""
        if self.model.hybrid:
            return iops.linear_f32(h, self.lm_head.weight)
        return ops.linear(h, self.head_weight()).float()

    @torch.no_grad()
    def _decode_steps(self, input_ids, max_new_tokens=64, do_sample=False, temperature=1.0, top_k=0, top_p=0.0,
                      eos_token_id=None, repetition_penalty=1.0, stop_words_ids=None, soft_prefix=None,
                      attention_mask=None, cuda_graph=True, **_):
        """Greedy / sampled decoding from the cache / state manager; yields the running ``[b, s]`` token tensor after
        every new token.  ``attention_mask``: rows of unequal length (padding on either side of ``input_ids``; new
        tokens are appended after column ``s``).  A row ends at ``eos_token_id`` or when its tail equals one of
        ``stop_words_ids`` (token sequences; the stop sequence stays in the output, later positions are filled with eos).
        ``cuda_graph``: on a GPU, replay the decode step as a CUDA graph once it has run eagerly (not with dynamic NTK,
        whose tables depend on the length, nor with the 8-bit cache).
        ``soft_prefix``: ``{"embeds": [P, hidden]}`` (prompt tuning: virtual input embeddings in front of the
        prompt) or ``{"kv": [layers, 2, P, kv_heads, head_dim]}`` (prefix tuning: pre-filled cache entries)."""
        from ...infer.generation import sample_next
        a = self.arch
        eos = a.eos_token_id if eos_token_id is None else eos_token_id
        stops = [torch.tensor(w, dtype=torch.long, device=input_ids.device) for w in (stop_words_ids or []) if len(w)]
        b, s = input_ids.shape
        dev, dt = input_ids.device, self.lm_head.weight.dtype
        real = torch.ones(b, s, dtype=torch.bool) if attention_mask is None else attention_mask.bool().cpu()
        prompts = [input_ids[i][real[i].to(dev)] for i in range(b)]
        soft = soft_prefix or {}
        pre_kv = soft.get("kv")
        pre_emb = soft.get("embeds")
        n_kv = 0 if pre_kv is None else pre_kv.shape[2]
        n_emb = 0 if pre_emb is None else pre_emb.shape[0]
        if (n_kv or n_emb) and self.model.keeps_tokens:
            raise NotImplementedError(f"{a.family}: soft prefixes (the embedding depends on token pairs)")
        state = self.new_state(b, s + max_new_tokens + n_kv + n_emb)
        slots = [state.open() for _ in range(b)]
        if n_kv:
            for l, c in enumerate(state.layers):
                k0, v0 = (pre_kv[l, i].to(dt) for i in (0, 1))
                if isinstance(c, dict):
                    c["kq"].append(0, k0.unsqueeze(0).expand(b, -1, -1, -1))
                    c["vq"].append(0, v0.unsqueeze(0).expand(b, -1, -1, -1))
                    c["len"] = n_kv
                else:
                    c.load_prefix(slots, k0, v0)
            for i in slots:
                state.lengths[i] = n_kv
        if a.use_cache_quantization and (not bool(real.all()) or slots != list(range(b))):
            raise ValueError("the 8-bit cache holds a dense batch: prompts of one length only")
        embeds = None
        if n_emb:
            embeds = torch.cat([torch.cat((pre_emb.to(dt), self.model.embed_tokens(p))) for p in prompts])
            prompts = [torch.cat((p.new_zeros(n_emb), p)) for p in prompts]      # shapes only: the embeddings are given
        toks = input_ids
        seen_mask = real.to(dev)
        done = torch.zeros(b, dtype=torch.bool, device=dev)
        fill = eos if eos is not None else 0
        graph = None
        for step in range(max_new_tokens):
            if step == 0:
                h, meta = self.step(state, slots, prompts, inputs_embeds=embeds)
                h = h[meta["last_rows"].to(h.device)]
                logits = self.logits(h)
            elif graph is not None:
                logits = graph.step(toks[:, -1])
            else:
                logits = self.logits(self.step(state, slots, toks[:, -1])[0])
                if cuda_graph and dev.type == "cuda" and dt != torch.float16 and not a.use_cache_quantization and \
                        a.rope_dynamic_ntk_max_pos is None and max_new_tokens - step > 4:
                    graph = DecodeGraph(self, state, slots)
            if repetition_penalty != 1.0:
                seen = torch.gather(logits, 1, toks)
                pen = torch.where(seen > 0, seen / repetition_penalty, seen * repetition_penalty)
                logits = logits.scatter(1, toks, torch.where(seen_mask, pen, seen)) if bool(real.all()) else \
                    _penalise(logits, toks, seen_mask, pen)
            nxt = sample_next(logits, temperature, top_k, top_p, greedy=not do_sample)
            if eos is not None or stops:
                nxt = torch.where(done, torch.full_like(nxt, fill), nxt)
            toks = torch.cat((toks, nxt.unsqueeze(1)), 1)
            seen_mask = F.pad(seen_mask, (0, 1), value=True)
            if eos is not None:
                done |= nxt == eos
            new_len = toks.shape[1] - s
            for w in stops:
                if new_len >= len(w):
                    done |= (toks[:, -len(w):] == w).all(dim=1)
            yield toks
            if (eos is not None or stops) and bool(done.all()):
                break

    def generate(self, input_ids, attention_mask=None, max_new_tokens=64, num_beams=1, **kw):
        toks = input_ids
        for toks in self._decode_steps(input_ids, max_new_tokens=max_new_tokens, attention_mask=attention_mask, **kw):
            pass
        return toks

    def generate_stream(self, input_ids, max_new_tokens=64, **kw):
        """Yields the newest token of every row (``[b]``) as soon as it is decoded."""
        for toks in self._decode_steps(input_ids, max_new_tokens=max_new_tokens, **kw):
            yield toks[:, -1]

    # ---- checkpoint IO --------------------------------------------------------------------------------
    def canonical_state(self):
        return {k: v for k, v in self.state_dict().items()}

    def save_pretrained(self, path, state_dict=None, family_format=True, safe_serialization=False, **_):
        from .io import export_state
        os.makedirs(path, exist_ok=True)
        sd = state_dict if state_dict is not None else self.state_dict()
        sd = export_state({k: v.detach().cpu() for k, v in sd.items()}, self.arch) if family_format else sd
        torch.save(sd, os.path.join(path, "pytorch_model.bin"))
        from .io import export_config
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(export_config(self.arch), f, indent=2)

    @classmethod
    def from_pretrained(cls, path, family=None, torch_dtype=torch.float32, arch_overrides=None, **_):
        from .io import import_state, sizes_from_state
        from ...ckpt.hf_import import load_hf_state
        with open(os.path.join(path, "config.json")) as f:
            cfg = json.load(f)
        arch = arch_from_hf_config(cfg, family)
        raw = load_hf_state(path)
        sizes_from_state(arch, raw)
        for k, v in (arch_overrides or {}).items():
            setattr(arch, k, v)
        if isinstance(torch_dtype, str):
            torch_dtype = getattr(torch, torch_dtype.replace("torch.", ""))
        model = cls(arch, torch_dtype)
        sd = import_state(raw, arch)
        missing, unexpected = model.load_state_dict(sd, strict=False)      # copies into each parameter's own dtype
        missing = [m for m in missing if not (arch.tie_word_embeddings and m == "lm_head.weight")]
        if missing or unexpected:
            raise RuntimeError(f"from_pretrained({path}): missing {missing[:8]}, unexpected {unexpected[:8]}")
        if arch.tie_word_embeddings:
            model.lm_head.weight = model.model.embed_tokens.weight
        return model
