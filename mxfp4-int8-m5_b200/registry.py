"""Model registry: from a model folder (config.json + model.safetensors) to the framework's prefill and decode classes.

An architecture is found by config.json's "architecture" or "model_type".  Each entry builds the pair (prefill, decode) that the
rest of the framework works with: prefill.make_cache / hidden / logits over portions of a sequence, decode.step / generate."""
import json
import os
from dataclasses import dataclass

import torch

from . import _lib
from . import build as _build
from . import decode as DEC
from . import fused_hybrid as FH
from . import fused_olmoe as FO
from . import fused_qwen3 as FQ
from . import host_model as HM


class UnsupportedType(TypeError):
    """The architecture has no kernels for the requested number format."""


@dataclass
class Bundle:
    """A loaded model: its name, prefill and decode objects, vocabulary size, and the check for waits that ran out."""
    name: str
    prefill: object
    decode: object
    vocab_size: int
    check_status: object


def read_safetensors(path, device="cpu"):
    """{name: tensor} of one safetensors file."""
    from safetensors.torch import load_file
    return load_file(path, device=str(device))


def _weights(path, device):
    files = sorted(f for f in os.listdir(path) if f.endswith(".safetensors"))
    if not files:
        raise FileNotFoundError(f"no .safetensors file in {path}")
    sd = {}
    for f in files:
        sd.update(read_safetensors(os.path.join(path, f), device))
    return sd


def _hybrid(cfg, path, dtype, device):
    _build.build(which="mixers")
    args = HM.HybridArgs.from_config(cfg)
    model = HM.HybridLM(args, device, dtype).load_state_dict(_weights(path, device))
    fused = FH.FusedHybrid(model)
    return Bundle(args.model_type, fused, DEC.DecodeHybrid(fused), args.vocab_size, _lib.check_mixer_status)


def _hf_args(cfg):
    return HM.ModelArgs(cfg["hidden_size"], cfg["intermediate_size"], cfg["num_hidden_layers"], cfg["num_attention_heads"],
                        cfg["num_key_value_heads"], cfg.get("head_dim") or cfg["hidden_size"] // cfg["num_attention_heads"],
                        cfg["rms_norm_eps"], cfg.get("rope_theta", 1e4), cfg["vocab_size"], cfg.get("tie_word_embeddings", False),
                        cfg.get("num_experts", 0), cfg.get("num_experts_per_tok", 0), cfg.get("norm_topk_prob", False), cfg["model_type"])


def _w4a8(cfg, path, dtype, device):
    if dtype != torch.bfloat16:
        raise UnsupportedType(f"{cfg['model_type']} runs with packed 4-bit weights and bfloat16 activations, not {dtype}")
    _build.build(which="scmx")
    args = _hf_args(cfg)
    with torch.device(device):
        model = HM.CausalLM(args)
    model.load_hf_state_dict(_weights(path, device))
    if args.num_experts:
        fused = FO.FusedOlmoe(model, FO.pack_olmoe(model, on_device=True))
        return Bundle(args.model_type, fused, DEC.DecodeOlmoe(fused), args.vocab_size, _lib.check_status)
    fused = FQ.FusedQwen3(model, FQ.pack_model(model, on_device=True))
    return Bundle(args.model_type, fused, DEC.DecodeQwen3(fused), args.vocab_size, _lib.check_status)


ARCHITECTURES = {**{name: _hybrid for name in HM.DESIGNS}, "qwen3": _w4a8, "olmoe": _w4a8}


def architecture(cfg):
    """Registry key of a config.json dictionary."""
    name = str(cfg.get("architecture") or cfg.get("model_type") or "").lower()
    if name not in ARCHITECTURES:
        raise KeyError(f"architecture {name!r} is not registered ({', '.join(sorted(ARCHITECTURES))})")
    return name


def load(path, dtype=torch.bfloat16, device="cuda"):
    """Loads the model in folder `path`; builds the kernel library that it needs if a source is newer."""
    with open(os.path.join(path, "config.json")) as fh:
        cfg = json.load(fh)
    return ARCHITECTURES[architecture(cfg)](cfg, path, dtype, device)
