"""Model registry: from a folder with ``config.json`` and safetensors weights to the engine that serves it.

``load_engine`` looks the architecture up, builds the kernel library that this engine uses if it is not
built yet, reads the weights and constructs the engine. A new design registers a ``ModelEntry``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Sequence

import torch

from . import build
from .checkpoint import TensorBag, read_config, read_weights

DTYPES = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32}


@dataclass(frozen=True)
class ModelEntry:
    library: str                                   # of build.LIBRARIES
    dtypes: Sequence[str]                          # storage types, the default first
    construct: Callable                            # (config dict, tensors, device, dtype, max_seq_len, **kw) -> engine


_MODELS: dict[str, ModelEntry] = {}


def register(name: str, entry: ModelEntry) -> None:
    _MODELS[name] = entry


def architectures() -> list[str]:
    return sorted(_MODELS)


def architecture_of(config: dict) -> str:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in _MODELS:
        raise ValueError(f"architecture {name!r} is not one of {architectures()}")
    return name


def supports(config: dict, dtype: str) -> bool:
    return dtype in _MODELS[architecture_of(config)].dtypes


def load_engine(model_dir: str, device="cuda:0", dtype: str | None = None, max_seq_len: int = 4096, **kw):
    config = read_config(model_dir)
    entry = _MODELS[architecture_of(config)]
    dtype = dtype or entry.dtypes[0]
    if dtype not in entry.dtypes:
        raise ValueError(f"{architecture_of(config)} runs in {', '.join(entry.dtypes)}, not {dtype}")
    build.build_library(entry.library)
    if not torch.cuda.is_available():
        raise RuntimeError("leankv_b200 runs only on the GPU (no CPU fallback)")
    return entry.construct(config, read_weights(model_dir), torch.device(device), DTYPES[dtype], max_seq_len, **kw)


# ── the models ───────────────────────────────────────────────────────────────────────────────

def _mixer_model(config, tensors, device, dtype, max_seq_len, **kw):
    from .mixer_engine import MixerDecodeEngine, MixerModelConfig

    return MixerDecodeEngine(MixerModelConfig.from_dict(config), tensors, device, max_seq_len=max_seq_len, dtype=dtype,
                             **kw)


def _llama_model(config, tensors, device, dtype, max_seq_len, **kw):
    """Llama / Mistral checkpoints under their usual tensor names, served by the TEAL + TurboQuant engine."""
    from types import SimpleNamespace

    from .engine import PROJ_NAMES, DecodeEngine, DecoderConfig

    cfg = DecoderConfig.from_hf(SimpleNamespace(**config))
    bag = TensorBag(tensors)
    H, V, I = cfg.hidden_size, cfg.vocab_size, cfg.intermediate_size
    q, kv = cfg.num_q_heads * cfg.head_dim, cfg.num_kv_heads * cfg.head_dim
    shapes = {"q_proj": (q, H), "k_proj": (kv, H), "v_proj": (kv, H), "o_proj": (H, q),
              "gate_proj": (I, H), "up_proj": (I, H), "down_proj": (H, I)}
    put = lambda t: t.to(device, dtype)
    full = {"embed": put(bag.take("model.embed_tokens.weight", V, H)),
            "final_norm": put(bag.take("model.norm.weight", H)), "layers": []}
    full["lm_head"] = full["embed"] if config.get("tie_word_embeddings") else put(bag.take("lm_head.weight", V, H))
    for i in range(cfg.num_layers):
        p = f"model.layers.{i}."
        lw = {"ln1": put(bag.take(p + "input_layernorm.weight", H)),
              "ln2": put(bag.take(p + "post_attention_layernorm.weight", H))}
        for name in PROJ_NAMES:
            part = "self_attn" if name in ("q_proj", "k_proj", "v_proj", "o_proj") else "mlp"
            lw[name] = put(bag.take(f"{p}{part}.{name}.weight", *shapes[name]))
        full["layers"].append(lw)
    return DecodeEngine(cfg, DecodeEngine.shard_weights(full, cfg, 0, 1), device, max_seq_len=max_seq_len, **kw)


for _name in ("Rorosun", "Pefitar"):
    register(_name, ModelEntry("libleankv_mixers.so", ("bfloat16", "float32"), _mixer_model))
for _name in ("LlamaForCausalLM", "MistralForCausalLM"):
    register(_name, ModelEntry("libleankv_b200.so", ("float16",), _llama_model))
