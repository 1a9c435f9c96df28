"""Fizesun: latent attention with a rotated part and head gates, dense xIELU and clamped-gate expert feed-forwards, one residual stream
with a one-number RMS norm and an input convolution before every sublayer, and a range of layers that runs several times.

Reads a checkpoint directory's ``config.json`` and ``model.safetensors`` into the generic hybrid configuration and weights
(models/hybrid.py).  Every size and constant comes from the configuration or a tensor's shape.
"""
from __future__ import annotations

from .hybrid import (HybridConfig, HybridLayer, HybridWeights, LatentSpec, LayerSpec, LoopSpec, MlpSpec, MoeSpec, pack_gated_moe, pack_input_conv,
                     pack_latent, pack_loop_in, pack_plain_mlp, pad_cols, xielu)
from ..ops.hybrid import RmsNorm


def read_config(doc: dict, name: str = "fizesun") -> HybridConfig:
    layers = []
    for i, entry in enumerate(doc["layers"]):
        m, mlp = entry["mixer"], entry.get("mlp")
        if entry["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        rot, dims = m.get("rot") or {}, int(m.get("rot_dim", 0))
        if int(rot.get("dims", dims)) != dims:
            raise ValueError(f"layer {i}: {rot['dims']} of {dims} rotated dimensions turn; all of them do in this design")
        mixer = LatentSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), rank=int(m["kv_rank"]), scale=float(m["scale"]), rot_dim=dims,
                           rot_base=float(rot.get("base", 1.0)), gated=True)
        ff = None
        if mlp is not None and mlp["kind"] == "dense":
            ff = MlpSpec(int(mlp["ff"]), "xielu")
        elif mlp is not None and mlp["kind"] == "moe":
            shared = mlp.get("shared") or {}
            ff = MoeSpec(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), inter=int(mlp["expert"]["ff"]), renormalize=True,
                         act="clamp_glu", limit=float(mlp["expert"]["limit"]), shared_inter=int(shared.get("ff", 0)),
                         shared_limit=float(shared.get("limit", 0.0)), bias=True)
        elif mlp is not None:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        layers.append(LayerSpec(mixer, ff))
    loop = doc.get("loop")
    cfg = HybridConfig(vocab=int(doc["vocab"]), hidden=int(doc["width"]), layers=layers, norm_eps=float(doc["norm"]["eps"]), name=name, residual="pre",
                       input_taps=int(doc["canon"]["taps"]), loop=LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)
    cfg.validate()
    return cfg


def load_weights(cfg: HybridConfig, tensors, dtype, device) -> HybridWeights:
    """``tensors``: name -> CPU tensor mapping (package/safetensors.py reads the file)."""
    used = set()

    def take(name, f32=False):
        used.add(name)
        t = tensors[name].to(device)
        return t.float() if f32 else t.to(dtype)

    def norm(name):                # one number for all coordinates
        return RmsNorm(take(name, True).reshape(1).expand(cfg.hidden).contiguous(), cfg.norm_eps)

    w = HybridWeights(embed=take("embed"), embed_norm=norm("embed.norm"))
    if cfg.loop is not None:
        w.loop_in, w.loop_step = pack_loop_in(take("loop.in")), take("loop.step", True).contiguous()
    for i, spec in enumerate(cfg.layers):
        p, f = f"l{i}.", spec.mlp
        x = lambda name, f32=False: take(p + "mix." + name, f32)
        mixer = pack_latent(spec.mixer, x("q"), x("dkv"), x("dkv.norm", True), x("uk"), x("uv"), x("o"), x("g"))
        layer = HybridLayer(norm1=norm(p + "norm1"), hc1=None, mixer=mixer, conv1=pack_input_conv(take(p + "canon1", True)))
        if f is not None:
            layer.norm2, layer.conv2 = norm(p + "norm2"), pack_input_conv(take(p + "canon2", True))
        y = lambda name, f32=False: take(p + "mlp." + name, f32)
        if isinstance(f, MoeSpec):
            part = lambda kind: [y(f"e{e}.{kind}") for e in range(f.experts)]
            shared = tuple(y("shared." + n) for n in ("gate", "up", "down", "sg")) if f.shared_inter else None
            layer.moe = pack_gated_moe(y("router"), y("router.b", True), part("gate"), part("up"), part("down"), shared)
        elif f is not None:
            pack_plain_mlp(layer, y("up"), y("down"), xielu(*y("act", True).tolist()))
        w.layers.append(layer)
    w.final_norm, w.lm_head = norm("final.norm"), pad_cols(take("head"))
    w.unused = sorted(set(tensors) - used)
    return w
