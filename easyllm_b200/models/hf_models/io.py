"""Family ↔ canonical (HF Llama names) state-dict and config translation for ``hf_models``.

The reference vendors one modeling file per family with its own parameter names
(llm/models/hf_models/qwen/modeling_qwen.py ``c_attn`` / ``w1`` / ``w2``, internlm2/modeling_internlm2.py
interleaved ``wqkv``, baichuan*/modeling_baichuan.py ``W_pack``); here one decoder serves all of them and this
module maps their checkpoints in and out."""
from __future__ import annotations

import torch

from ...ckpt.hf_import import canonicalize
from .feedforward import SparseGLU

_FAMILY_RULES = {"llama": "llama", "internlm": "llama", "baichuan": "baichuan", "baichuan2": "baichuan",
                 "baichuan2-13b": "baichuan", "internlm2": "internlm2", "qwen": "qwen", "pafodra": "pafodra",
                 "megozen": "megozen"}
_MIXES = "rkvgw"          # rows of TimeMix.mu


def import_state(hf_state, arch):
    """Any family's on-disk names → ``model.layers.N.self_attn.q_proj.weight`` style names."""
    canon = canonicalize(hf_state, _FAMILY_RULES[arch.family], arch.num_attention_heads, arch.kv_heads, arch.hidden_size)
    out = {}
    for slot, tensors in canon.items():
        for name, t in tensors.items():
            if slot == "embed":
                out["model.embed_pairs.weight" if name == "pairs" else "model.embed_tokens.weight"] = t
            elif slot == "norm":
                out[f"model.norm.{name}"] = t
            elif slot == "head":
                out["lm_head.weight"] = t
            else:
                out[f"model.layers.{slot}.{name}"] = t
    return _stack_hybrid(out, arch) if arch.layers is not None else out


def sizes_from_state(arch, raw):
    """Sizes that only the tensors tell (ranks of the low-rank projections) → the arch's layer specs."""
    from .modeling import weight_owner
    for i, spec in enumerate(arch.layers or []):
        n = f"l{weight_owner(arch.layers, i)}.mix"
        if spec.type == "wkv":
            spec.mixer["decay_rank"] = raw[n + ".w1"].shape[0]
        elif spec.type == "channel_delta":
            spec.mixer["decay_rank"], spec.mixer["gate_rank"] = raw[n + ".a1"].shape[0], raw[n + ".g1"].shape[0]


def _stack_hybrid(sd, arch):
    """Per-expert and per-mix tensors stacked as the modules hold them, and the tensors of a layer repeated under the
    index of every layer that uses them (``nn.Module.state_dict`` lists a shared module at each of its places)."""
    from .modeling import weight_owner
    out = {}
    for i, spec in enumerate(arch.layers):
        src, dst = f"model.layers.{weight_owner(arch.layers, i)}.", f"model.layers.{i}."
        mine = {k[len(src):]: v for k, v in sd.items() if k.startswith(src)}
        if spec.type == "wkv":
            mine["mixer.mu"] = torch.stack([mine.pop(f"mixer.mu.{c}") for c in _MIXES])
        if spec.mlp is None:
            mine.pop("mlp_layernorm.weight", None)          # the norm of a feed-forward that is not there
        if spec.mlp is not None and spec.mlp["kind"] == "moe":
            if arch.expert_form == "glu":
                mine["mlp.experts_gate_up"] = torch.stack([SparseGLU.blocked(*(mine.pop(f"mlp.experts.{e}.{p}") for p in ("gate", "up")))
                                                           for e in range(spec.mlp["router"]["experts"])])
            for p in ("down",) if arch.expert_form == "glu" else ("up", "down"):
                mine[f"mlp.experts_{p}"] = torch.stack([mine.pop(f"mlp.experts.{e}.{p}")
                                                        for e in range(spec.mlp["router"]["experts"])])
        out.update({dst + k: v for k, v in mine.items()})
    out.update({k: v for k, v in sd.items() if not k.startswith("model.layers.")})
    return out


def _export_hybrid(sd, arch):
    from .modeling import weight_owner
    from ...ckpt.hf_import import HYBRID_NAMES
    back = {v: k for k, v in HYBRID_NAMES[arch.family].items()}
    out = {"embed": sd["model.embed_tokens.weight"], "head": sd["lm_head.weight"]}
    if arch.bigram is not None:
        out["bigram"] = sd["model.embed_pairs.weight"]
    for n, suffix in (("weight", ""), ("bias", ".b"), ("alpha", ".alpha")):
        if "model.norm." + n in sd:
            out["final.norm" + suffix] = sd["model.norm." + n]
    for i in range(len(arch.layers)):
        if weight_owner(arch.layers, i) != i:
            continue
        pre = f"model.layers.{i}."
        for k, v in sd.items():
            if not k.startswith(pre):
                continue
            name = k[len(pre):]
            if name == "mixer.mu":
                out.update({f"l{i}.mix.mu.{c}": v[j] for j, c in enumerate(_MIXES)})
            elif name == "mlp.experts_gate_up":
                for e, w in enumerate(v):
                    out[f"l{i}.mlp.e{e}.gate"], out[f"l{i}.mlp.e{e}.up"] = SparseGLU.split(w)
            elif name in ("mlp.experts_up", "mlp.experts_down"):
                out.update({f"l{i}.mlp.e{e}.{name[12:]}": w for e, w in enumerate(v)})
            else:
                out[f"l{i}.{back[name]}"] = v
    return {k: v.contiguous() for k, v in out.items()}


def export_state(sd, arch):
    """Canonical names → the family's on-disk names (inverse of ``import_state``)."""
    fam = arch.family
    if fam in ("llama", "internlm"):
        return sd
    if arch.layers is not None:
        return _export_hybrid(sd, arch)
    out = {}
    L = arch.num_hidden_layers
    hq, hk, d, h = arch.num_attention_heads, arch.kv_heads, arch.head_dim, arch.hidden_size

    def layer(i, name):
        return sd[f"model.layers.{i}.{name}"]
    if fam.startswith("baichuan"):
        for k, v in sd.items():
            if ".self_attn.q_proj." in k or ".self_attn.k_proj." in k or ".self_attn.v_proj." in k:
                continue
            out[k] = v
        for i in range(L):
            out[f"model.layers.{i}.self_attn.W_pack.weight"] = torch.cat(
                [layer(i, f"self_attn.{p}_proj.weight") for p in "qkv"], 0)
        return out
    if fam == "internlm2":
        out["model.tok_embeddings.weight"] = sd["model.embed_tokens.weight"]
        out["model.norm.weight"] = sd["model.norm.weight"]
        out["output.weight"] = sd["lm_head.weight"]
        gs = hq // hk
        for i in range(L):
            q = layer(i, "self_attn.q_proj.weight").view(hk, gs, d, h)
            k = layer(i, "self_attn.k_proj.weight").view(hk, 1, d, h)
            v = layer(i, "self_attn.v_proj.weight").view(hk, 1, d, h)
            out[f"model.layers.{i}.attention.wqkv.weight"] = torch.cat((q, k, v), 1).reshape(-1, h)
            out[f"model.layers.{i}.attention.wo.weight"] = layer(i, "self_attn.o_proj.weight")
            out[f"model.layers.{i}.feed_forward.w1.weight"] = layer(i, "mlp.gate_proj.weight")
            out[f"model.layers.{i}.feed_forward.w3.weight"] = layer(i, "mlp.up_proj.weight")
            out[f"model.layers.{i}.feed_forward.w2.weight"] = layer(i, "mlp.down_proj.weight")
            out[f"model.layers.{i}.attention_norm.weight"] = layer(i, "input_layernorm.weight")
            out[f"model.layers.{i}.ffn_norm.weight"] = layer(i, "post_attention_layernorm.weight")
        return out
    if fam == "qwen":
        out["transformer.wte.weight"] = sd["model.embed_tokens.weight"]
        out["transformer.ln_f.weight"] = sd["model.norm.weight"]
        out["lm_head.weight"] = sd["lm_head.weight"]
        for i in range(L):
            out[f"transformer.h.{i}.attn.c_attn.weight"] = torch.cat([layer(i, f"self_attn.{p}_proj.weight") for p in "qkv"], 0)
            out[f"transformer.h.{i}.attn.c_attn.bias"] = torch.cat([layer(i, f"self_attn.{p}_proj.bias") for p in "qkv"], 0)
            out[f"transformer.h.{i}.attn.c_proj.weight"] = layer(i, "self_attn.o_proj.weight")
            out[f"transformer.h.{i}.mlp.w2.weight"] = layer(i, "mlp.gate_proj.weight")
            out[f"transformer.h.{i}.mlp.w1.weight"] = layer(i, "mlp.up_proj.weight")
            out[f"transformer.h.{i}.mlp.c_proj.weight"] = layer(i, "mlp.down_proj.weight")
            out[f"transformer.h.{i}.ln_1.weight"] = layer(i, "input_layernorm.weight")
            out[f"transformer.h.{i}.ln_2.weight"] = layer(i, "post_attention_layernorm.weight")
        return out
    raise ValueError(fam)


def export_config(arch):
    a = arch
    if a.layers is not None:
        layers = []
        for l in a.layers:
            e = {"type": l.type, "mixer": {k: v for k, v in l.mixer.items() if k not in ("decay_rank", "gate_rank")}, "mlp": l.mlp}
            layers.append(e if l.weights_of is None else dict(e, weights_of=l.weights_of))
        emb = {"scale": a.embedding_scale} if a.family == "pafodra" else {} if a.bigram is None else {"bigram": a.bigram}
        return {"architecture": a.family.capitalize(), "vocab": a.vocab_size, "width": a.hidden_size, "layers": layers,
                "norm": {"eps": a.norm_eps}, "embedding": emb}
    if a.family == "qwen":
        return {"model_type": "qwen", "vocab_size": a.vocab_size, "hidden_size": a.hidden_size,
                "intermediate_size": 2 * a.intermediate_size, "num_hidden_layers": a.num_hidden_layers,
                "num_attention_heads": a.num_attention_heads, "layer_norm_epsilon": a.rms_norm_eps,
                "rotary_emb_base": a.rope_theta, "use_logn_attn": a.use_logn_attn, "seq_length": a.seq_length,
                "use_cache_quantization": a.use_cache_quantization,
                "use_dynamic_ntk": a.rope_dynamic_ntk_max_pos is not None,
                "max_position_embeddings": a.max_position_embeddings}
    cfg = {"model_type": a.family, "vocab_size": a.vocab_size, "hidden_size": a.hidden_size,
           "intermediate_size": a.intermediate_size, "num_hidden_layers": a.num_hidden_layers,
           "num_attention_heads": a.num_attention_heads, "num_key_value_heads": a.kv_heads,
           "rms_norm_eps": a.rms_norm_eps, "rope_theta": a.rope_theta,
           "max_position_embeddings": a.max_position_embeddings, "tie_word_embeddings": a.tie_word_embeddings,
           "pad_token_id": a.pad_token_id, "bos_token_id": a.bos_token_id, "eos_token_id": a.eos_token_id}
    if a.family in ("internlm", "internlm2"):
        cfg["bias"] = a.qkv_bias
    if a.family == "llama":
        cfg["attention_bias"] = a.qkv_bias
        cfg["architectures"] = ["LlamaForCausalLM"]
    if a.rope_scaling_factor != 1.0:
        cfg["rope_scaling"] = {"type": "dynamic" if a.rope_dynamic_ntk_max_pos else "linear", "factor": a.rope_scaling_factor}
    return cfg
