"""Models by their configuration file: `load_model(device, folder)` reads config.json, chooses the builder registered for its
architecture and loads the folder's safetensors.  The reference has one constructor per model and no file form
(NN.Llama / NN.Phi3, src/NN.jl:417-507; weights by load_weights!, src/Weights.jl:60-114)."""
from __future__ import annotations

import json
import os

from .session import LayeredModel, Model
from .weights import load_safetensors

REGISTRY = {}


def register(*names):
    """Registers a builder (device, config, dtype) -> model for the architecture names of a config.json."""
    def add(fn):
        for n in names:
            REGISTRY[n] = fn
        return fn
    return add


def read_config(path):
    with open(os.path.join(path, "config.json")) as f:
        return json.load(f)


def architecture(config):
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in REGISTRY:
        raise ValueError(f"architecture {name!r} is not registered (known: {', '.join(sorted(REGISTRY))})")
    return name


def build_model(device, config, dtype="bf16"):
    return REGISTRY[architecture(config)](device, config, dtype)


def load_model(device, path, dtype="bf16"):
    """The model of a folder (config.json + *.safetensors).  A tensor the configuration needs and no file has is an error."""
    model = build_model(device, read_config(path), dtype)
    load_safetensors(model, path, warn_missing=False)
    missing = model.missing_weights()
    if missing:
        model.close()
        raise ValueError(f"{path}: no weights for {', '.join(missing[:8])}" + (" ..." if len(missing) > 8 else ""))
    return model


@register("LlamaForCausalLM")
def llama(device, config, dtype):
    return Model(device, n_layers=config["num_hidden_layers"], hidden=config["hidden_size"], n_heads=config["num_attention_heads"],
                 n_kv_heads=config.get("num_key_value_heads") or config["num_attention_heads"], intermediate=config["intermediate_size"],
                 vocab=config["vocab_size"], eps=config["rms_norm_eps"], rope_base=config.get("rope_theta", 10000.0), dtype=dtype)


def gibutar_layers(config):
    """Layer descriptions (LayeredModel) of a Gibutar configuration.  Fixed by the design: latent attention rotates interleaved
    pairs, retention rotates half-split pairs, the feed-forward is down(relu(up h)^2)."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        mx, mlp = layer["mixer"], layer.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: feed-forward of kind {mlp['kind']!r}")
        rot = mx.get("rot") or {}
        d = dict(mixer=layer["type"], heads=mx["heads"], dim=mx["dim"], vdim=mx["vdim"], ff=mlp["ff"] if mlp else 0,
                 rot_dims=rot.get("dims", 0), rot_base=rot.get("base", 1.0))
        if layer["type"] == "latent_attention":
            d.update(q_rank=mx["q_rank"], kv_rank=mx["kv_rank"], rot_dim=mx["rot_dim"], scale=mx["scale"], kv_from=mx.get("kv_from"),
                     rot_layout="interleaved")
        elif layer["type"] == "retention":
            d.update(decay=mx["decay"], rot_layout="half")
        else:
            raise ValueError(f"layer {i}: mixer {layer['type']!r}")
        layers.append(d)
    return layers


@register("Gibutar")
def gibutar(device, config, dtype):
    return LayeredModel(device, width=config["width"], vocab=config["vocab"], layers=gibutar_layers(config), eps=config["norm"]["eps"],
                        softcap=config.get("logit_softcap") or 0.0, dtype=dtype)
