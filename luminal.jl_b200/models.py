"""Models by their configuration file: `load_model(device, folder)` reads config.json, chooses the builder registered for its
architecture and loads the folder's safetensors.  The reference has one constructor per model and no file form
(NN.Llama / NN.Phi3, src/NN.jl:417-507; weights by load_weights!, src/Weights.jl:60-114)."""
from __future__ import annotations

import json
import os

from .session import LayeredModel, Model
from .weights import load_safetensors, safetensors_shapes

REGISTRY = {}


def register(*names):
    """Registers a builder (device, config, dtype, shapes) -> model for the architecture names of a config.json.  `shapes` (name ->
    shape of the weight file's tensors) is for sizes that no key of the configuration gives."""
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


def build_model(device, config, dtype="bf16", shapes=None):
    return REGISTRY[architecture(config)](device, config, dtype, shapes or {})


def load_model(device, path, dtype="bf16"):
    """The model of a folder (config.json + *.safetensors).  A tensor the configuration needs and no file has is an error."""
    model = build_model(device, read_config(path), dtype, safetensors_shapes(path))
    load_safetensors(model, path, warn_missing=False)
    missing = model.missing_weights()
    if missing:
        model.close()
        raise ValueError(f"{path}: no weights for {', '.join(missing[:8])}" + (" ..." if len(missing) > 8 else ""))
    return model


@register("LlamaForCausalLM")
def llama(device, config, dtype, shapes):
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
def gibutar(device, config, dtype, shapes):
    return LayeredModel(device, width=config["width"], vocab=config["vocab"], layers=gibutar_layers(config), eps=config["norm"]["eps"],
                        softcap=config.get("logit_softcap") or 0.0, dtype=dtype)


def kevatar_layers(config, shapes):
    """Layer descriptions (LayeredModel) of a Kevatar configuration.  Fixed by the design: rotations of interleaved pairs, unit key
    heads, the feed-forward down(silu(gate h) * up h).  The ranks of a channel-delta layer's decay and gate come from its tensors."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        mx, mlp, kind = layer["mixer"], layer.get("mlp"), layer["type"]
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: feed-forward of kind {mlp['kind']!r}")
        d = dict(mixer=kind, heads=mx["heads"], dim=mx["dim"], vdim=mx["vdim"], ff=mlp["ff"] if mlp else 0, ff_kind="silu_gate",
                 rot_layout="interleaved")
        if kind == "attention":
            rot = mx.get("rot") or {}
            d.update(kv_heads=mx["kv_heads"], scale=mx["scale"], score_cap=mx.get("softcap"), window=(mx.get("mask") or {}).get("size"),
                     kv_from=mx.get("kv_from"), rot_dims=rot.get("dims", 0), rot_base=rot.get("base"), rot_scaling=rot.get("scaling"))
        elif kind == "channel_delta":
            ranks = [shapes.get(f"l{i}.mix.{n}") for n in ("a1", "g1")]
            if None in ranks:
                raise ValueError(f"layer {i}: the shapes of l{i}.mix.a1 and l{i}.mix.g1 are needed for its ranks")
            d.update(kv_heads=mx["kv_heads"], conv=mx["conv"], decay_rank=ranks[0][0], gate_rank=ranks[1][0])
        elif kind == "lightning":
            d.update(decay=mx["decay"])
        else:
            raise ValueError(f"layer {i}: mixer {kind!r}")
        layers.append(d)
    return layers


@register("Kevatar")
def kevatar(device, config, dtype, shapes):
    return LayeredModel(device, width=config["width"], vocab=config["vocab"], layers=kevatar_layers(config, shapes), eps=config["norm"]["eps"],
                        block="postnorm", side_dim=(config.get("token_side") or {}).get("dim", 0), tied_head=True,
                        embed_scale=config["embedding"]["scale"], dtype=dtype)
