"""Sodurax: a decoder of attention layers on an fp32 residual stream, in which

  * every sublayer sits between two elementwise norms, x <- x + n_o(mixer(n_i(x))), x <- x + n_o'(ff(n_i'(x))), with
    n(z) = tanh(alpha z) w + b (no mean, no variance); the final norm is of the same kind;
  * attention has grouped key / value heads, biases on q, k and v, rotary positions on the first channels of a head with
    linearly interpolated positions, a sliding window beside which the first positions of the sequence stay visible, and a
    sigmoid output gate;
  * feed-forwards are routed: sigmoid scores, a learned correction per expert that only the choice sees, choice inside the
    best groups of neighbouring experts, weights that are not renormalised, ungated squared-ReLU experts;
  * a layer may run on the tensors of another one (`weights_of`), with a cache of its own;
  * the embedding table also makes the logits.

The model is the generic backbone (`transformer.py`) configured by `ModelConfig.layer_specs` (the layers that have tensors)
and `ModelConfig.layer_order` (the order they run in); this module only reads the family's `config.json` / tensor names.  A
checkpoint is `config.json` + `model.safetensors` with

    embed, final.norm{,.alpha,.b}, l<i>.{norm1,norm1b,norm2,norm2b}{,.alpha,.b}, l<i>.mix.{q,k,v}{,.b}, l<i>.mix.{g,o},
    l<i>.mlp.{router, correction, e<j>.{up,down}}
"""
from __future__ import annotations

import os
from typing import Dict, List

import torch

from .config import ExpertFFSpec, LayerSpec, MixerSpec, ModelConfig
from .transformer import TransformerLMHeadModel

__all__ = ["SoduraxForCausalLM", "sodurax_config", "convert_sodurax_state_dict", "load_sodurax", "stored_layers"]


class SoduraxForCausalLM(TransformerLMHeadModel):
    pass


def _owner(layers: List[dict], i: int) -> int:
    """The layer whose tensors layer i runs on."""
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError(f"layer {i}: `weights_of` runs in a circle")
        seen.add(i)
        i = layers[i]["weights_of"]
    return i


def stored_layers(hf: dict) -> List[int]:
    """Indices (into the config's layers) of the layers that have tensors of their own."""
    return [i for i, ly in enumerate(hf["layers"]) if ly.get("weights_of") is None]


def sodurax_config(hf: dict) -> ModelConfig:
    specs = []
    stored = stored_layers(hf)
    for i in stored:
        ly = hf["layers"][i]
        if ly["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {ly['type']!r}")
        m = ly["mixer"]
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        factor = float((rot.get("scaling") or {}).get("factor", 1.0))
        mixer = MixerSpec(kind="attention", heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"],
                          vdim=m.get("vdim", m["dim"]), bias=True, scale=m.get("scale"), rot_dims=rot.get("dims", 0),
                          rot_base=float(rot.get("base", 10000.0)), rot_scaling=None if factor == 1.0 else [factor],
                          window=mask.get("size", 0), keep_first=mask.get("keep_first", 0), out_gate=True, wide_weights=True)
        mlp = ly.get("mlp")
        if mlp is None:
            specs.append(LayerSpec(mixer=mixer))
        elif mlp.get("kind", "moe") == "moe":
            r = mlp["router"]
            groups = r.get("groups") or {}
            specs.append(LayerSpec(mixer=mixer, moe=ExpertFFSpec(
                experts=r["experts"], top=r["top"], ff=mlp["expert"]["ff"], act="relu2", score="sigmoid", correction=True,
                renormalize=False, groups=groups.get("count", 1), keep_groups=groups.get("keep", groups.get("count", 1)))))
        else:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    order = [stored.index(_owner(hf["layers"], i)) for i in range(len(hf["layers"]))]
    return ModelConfig(model_type="sodurax", vocab_size=hf["vocab"], hidden_size=hf["width"], intermediate_size=hf["width"],
                       layer_specs=specs, layer_order=None if order == list(range(len(specs))) else order,
                       norm_eps=hf["norm"]["eps"], norm_type="tanh", norm_placement="both", hidden_act="relu2", glu=False,
                       pos_type="none", fp32_residual=True, fp32_logits=True, tie_word_embeddings=True,
                       max_position_embeddings=1 << 20)


def convert_sodurax_state_dict(sd: Dict[str, torch.Tensor], cfg: ModelConfig, stored: List[int]) -> Dict[str, torch.Tensor]:
    """Checkpoint names -> backbone parameter names (`stored`: the checkpoint's index of every layer spec); q | k | v | output
    gate are stacked into one GEMM (the gate's rows have no bias), a layer's experts into batched tensors."""
    out = {"model.embed_tokens.weight": sd["embed"], "lm_head.weight": sd["embed"]}

    def norm(dst: str, src: str) -> None:
        out[dst + ".weight"], out[dst + ".bias"] = sd[src], sd[src + ".b"]
        out[dst + ".alpha"] = sd[src + ".alpha"].reshape(())

    norm("model.norm", "final.norm")
    for n, (i, spec) in enumerate(zip(stored, cfg.layer_specs)):
        src, dst, mx = f"l{i}.", f"model.layers.{n}.", spec.mixer
        norm(dst + "input_layernorm", src + "norm1")
        norm(dst + "mixer_out_norm", src + "norm1b")
        m, a = src + "mix.", dst + "self_attn."
        out[a + "qkv_proj.weight"] = torch.cat([sd[m + "q"], sd[m + "k"], sd[m + "v"], sd[m + "g"]], 0)
        out[a + "qkv_proj.bias"] = torch.cat([sd[m + "q.b"], sd[m + "k.b"], sd[m + "v.b"],
                                              torch.zeros_like(sd[m + "q.b"][:1]).expand(mx.heads * mx.vdim)], 0)
        out[a + "o_proj.weight"] = sd[m + "o"]
        if spec.moe is not None:
            norm(dst + "post_attention_layernorm", src + "norm2")
            norm(dst + "mlp_out_norm", src + "norm2b")
            p, q = src + "mlp.", dst + "mlp."
            out[q + "router.weight"], out[q + "correction"] = sd[p + "router"], sd[p + "correction"]
            out[q + "experts.w_up"] = torch.stack([sd[f"{p}e{e}.up"] for e in range(spec.moe.experts)])
            out[q + "experts.w_down"] = torch.stack([sd[f"{p}e{e}.down"] for e in range(spec.moe.experts)])
    return out


def load_sodurax(path: str, hf_cfg: dict, dtype: torch.dtype, device: str = "cpu") -> SoduraxForCausalLM:
    from safetensors.torch import load_file

    cfg = sodurax_config(hf_cfg)
    model = SoduraxForCausalLM(cfg)
    sd = convert_sodurax_state_dict(load_file(os.path.join(path, "model.safetensors")), cfg, stored_layers(hf_cfg))
    missing, unexpected = model.load_state_dict({k: v.to(torch.float32) for k, v in sd.items()}, strict=False)
    if missing or unexpected:
        raise RuntimeError(f"sodurax checkpoint does not fit the model: missing={missing[:6]} unexpected={unexpected[:6]}")
    model._pretrained_path = path
    return model.to(dtype).to(device)
