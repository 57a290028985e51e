"""Sumolorn: a pre-norm decoder on an fp32 residual stream whose layers, in any order given by its `config.json`, mix
tokens by

  * attention with grouped key / value heads, rotary positions on the first channels of a head (rotate-half pairs,
    frequencies slowed down by wavelength), soft-capped scores, a sliding window, a learned sink score per head and one
    sigmoid gate per head;
  * latent attention with a query latent, interleaved rotary pairs on the decoupled part, no window, a learned sink score
    and one sigmoid gate per head;
  * a PAIR: windowed attention whose q, k and v pass a short causal convolution (then positions, then unit-RMS q / k heads)
    beside gated linear attention (a decay per head and key channel); their outputs are RMS-normed and averaged.

Feed-forwards are clamped gated units or absent, norms are RMS norms with weights stored around zero, a span of layers may
run several times in a row (every pass with a cache and a state of its own), logits are scaled.

The model is the generic backbone (`transformer.py`) configured by `ModelConfig.layer_specs` (the layers that have tensors)
and `ModelConfig.layer_order` (the order they run in); this module only reads the family's `config.json` / tensor names.  A
checkpoint is `config.json` + `model.safetensors` with

    embed, head, final.norm, l<i>.norm1, l<i>.norm2, l<i>.mlp.{gate,up,down},
    l<i>.mix.{q,k,v,sink,g,o} or l<i>.mix.{dq{,.norm},uq,dkv{,.norm},uk,uv,sink,g,o} or
    l<i>.mix.left.{q{,.conv},k{,.conv},v{,.conv},o,out} + l<i>.mix.right.{q,k,v,g,o,norm,a1,a2{,.b},out}
"""
from __future__ import annotations

import os
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .config import LayerSpec, MixerSpec, ModelConfig
from .gopunex import read_safetensors_shapes
from .transformer import TransformerLMHeadModel

__all__ = ["SumolornForCausalLM", "sumolorn_config", "convert_sumolorn_state_dict", "load_sumolorn"]


class SumolornForCausalLM(TransformerLMHeadModel):
    pass


def _rot_fields(rot: dict, interleaved: bool) -> dict:
    sc = rot.get("scaling")
    return dict(rot_base=float(rot.get("base", 10000.0)), rot_interleaved=interleaved,
                rot_scaling=None if not sc else ["wavelength", float(sc["factor"]), float(sc["low"]), float(sc["high"]),
                                                 float(sc["original"])])


def _attention_fields(m: dict) -> dict:
    return dict(kind="attention", heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"],
                vdim=m.get("vdim", m["dim"]), scale=m.get("scale"), window=(m.get("mask") or {}).get("size", 0),
                softcap=float(m.get("softcap") or 0.0), rot_dims=(m.get("rot") or {}).get("dims", 0), wide_weights=True,
                **_rot_fields(m.get("rot") or {}, False))


def sumolorn_config(hf: dict, shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> ModelConfig:
    """`shapes` (tensor name -> shape, from the checkpoint's header) gives the one size the config leaves to the tensors: the
    rank of the decay projection."""
    shapes = shapes or {}
    specs = []
    for i, ly in enumerate(hf["layers"]):
        m, kind = ly["mixer"], ly["type"]
        if kind == "attention":
            mixer = MixerSpec(**_attention_fields(m), sink_learned=True, head_gate=True)
        elif kind == "latent_attention":
            mixer = MixerSpec(kind="latent", heads=m["heads"], kv_heads=1, dim=m["dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                              q_rank=m["q_rank"], rot_dim=m["rot_dim"], rot_dims=m["rot_dim"], scale=m.get("scale"),
                              sink_learned=True, head_gate=True, wide_weights=True, **_rot_fields(m.get("rot") or {}, True))
        elif kind == "parallel":
            lm, rm = m["left"], m["right"]
            rank = shapes.get(f"l{i}.mix.right.a1", (rm.get("rank", 16),))[0]
            left = MixerSpec(**_attention_fields(lm), conv=lm["conv"], conv_values=True, head_unit_norm=True)
            right = MixerSpec(kind="gla", heads=rm["heads"], dim=rm["dim"], vdim=rm.get("vdim", rm["dim"]),
                              tau=float(rm["tau"]), decay_rank=rank)
            mixer = MixerSpec(kind="pair", parts=[left, right])
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        mlp = ly.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        specs.append(LayerSpec(mixer=mixer) if mlp is None else
                     LayerSpec(mixer=mixer, ff=mlp["ff"], ff_act="clamped", ff_limit=float(mlp["limit"])))
    ffs = [s.ff for s in specs if s.ff is not None]
    return ModelConfig(model_type="sumolorn", vocab_size=hf["vocab"], hidden_size=hf["width"],
                       intermediate_size=max(ffs) if ffs else hf["width"], layer_specs=specs,
                       layer_order=_order(len(specs), hf.get("loop")), norm_eps=hf["norm"]["eps"], norm_type="rms",
                       norm_weight_offset=1.0, hidden_act="clamped", glu=True, pos_type="none", fp32_residual=True,
                       fp32_logits=True, logit_scale=float(hf.get("logit_scale", 1.0)), tie_word_embeddings=False,
                       max_position_embeddings=1 << 20)


def _order(layers: int, loop: Optional[dict]) -> Optional[List[int]]:
    """The layers in the order they run, None when that is each of them once."""
    if not loop:
        return None
    a, b = loop["start"], loop["stop"]
    order = list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, layers))
    return None if order == list(range(layers)) else order


def _stack(parts: Sequence[torch.Tensor], rows: int) -> torch.Tensor:
    """Projections that read the same input as one weight of `rows` rows (zero rows behind the last part)."""
    w = torch.cat(list(parts), 0)
    return torch.cat([w, w.new_zeros(rows - w.shape[0], w.shape[1])], 0)


def _convert_mixer(sd: Dict[str, torch.Tensor], m: str, a: str, mx: MixerSpec, own: Dict[str, Tuple[int, ...]],
                   out: Dict[str, torch.Tensor]) -> None:
    """Tensors `m + name` of one mixer -> parameters `a + name`; `own`: shapes of the model's parameters."""
    if mx.kind == "attention":
        rows = ["q", "k", "v"] + (["g"] if mx.head_gate else [])
        out[a + "qkv_proj.weight"] = _stack([sd[m + n] for n in rows], own[a + "qkv_proj.weight"][0])
        if mx.conv:
            out[a + "conv_weight"] = torch.cat([sd[m + n + ".conv"] for n in ("q", "k", "v")], 0)
        if mx.sink_learned:
            out[a + "sink_logit"] = sd[m + "sink"]
    elif mx.kind == "latent":
        out[a + "in_proj.weight"] = _stack([sd[m + n] for n in ("dq", "dkv", "g")], own[a + "in_proj.weight"][0])
        out[a + "dq_norm_weight"], out[a + "dkv_norm_weight"] = sd[m + "dq.norm"], sd[m + "dkv.norm"]
        out[a + "uq_proj.weight"] = sd[m + "uq"]
        out[a + "uk"] = sd[m + "uk"].reshape(mx.heads, mx.dim, mx.kv_rank)
        out[a + "uv"] = sd[m + "uv"].reshape(mx.heads, mx.vdim, mx.kv_rank)
        out[a + "sink_logit"] = sd[m + "sink"]
    else:
        out[a + "in_proj.weight"] = _stack([sd[m + n] for n in ("q", "k", "v", "g", "a1")], own[a + "in_proj.weight"][0])
        out[a + "decay_up.weight"], out[a + "decay_bias"] = sd[m + "a2"], sd[m + "a2.b"]
        out[a + "norm_weight"] = sd[m + "norm"]
    out[a + "o_proj.weight"] = sd[m + "o"]


def convert_sumolorn_state_dict(sd: Dict[str, torch.Tensor], model: SumolornForCausalLM) -> Dict[str, torch.Tensor]:
    """Checkpoint names -> `model`'s parameter names; projections that read the same input are stacked into one GEMM."""
    own = {n: tuple(p.shape) for n, p in model.named_parameters()}
    out = {"model.embed_tokens.weight": sd["embed"], "lm_head.weight": sd["head"], "model.norm.weight": sd["final.norm"]}
    for i, spec in enumerate(model.cfg.layer_specs):
        src, dst = f"l{i}.", f"model.layers.{i}."
        out[dst + "input_layernorm.weight"] = sd[src + "norm1"]
        if spec.ff is not None:
            out[dst + "post_attention_layernorm.weight"] = sd[src + "norm2"]
            out[dst + "mlp.gate_up_proj.weight"] = torch.cat([sd[src + "mlp.gate"], sd[src + "mlp.up"]], 0)
            out[dst + "mlp.down_proj.weight"] = sd[src + "mlp.down"]
        m, a, mx = src + "mix.", dst + "self_attn.", spec.mixer
        if mx.kind == "pair":
            for j, (side, part) in enumerate(zip(("left.", "right."), mx.parts)):
                _convert_mixer(sd, m + side, f"{a}parts.{j}.", part, own, out)
                out[f"{a}out_norm_weights.{j}"] = sd[m + side + "out"]
        else:
            _convert_mixer(sd, m, a, mx, own, out)
    return out


def load_sumolorn(path: str, hf_cfg: dict, dtype: torch.dtype, device: str = "cpu") -> SumolornForCausalLM:
    from safetensors.torch import load_file

    st = os.path.join(path, "model.safetensors")
    model = SumolornForCausalLM(sumolorn_config(hf_cfg, read_safetensors_shapes(st)))
    sd = convert_sumolorn_state_dict(load_file(st), model)
    missing, unexpected = model.load_state_dict({k: v.to(torch.float32) for k, v in sd.items()}, strict=False)
    if missing or unexpected:
        raise RuntimeError(f"sumolorn checkpoint does not fit the model: missing={missing[:6]} unexpected={unexpected[:6]}")
    model._pretrained_path = path
    return model.to(dtype).to(device)
