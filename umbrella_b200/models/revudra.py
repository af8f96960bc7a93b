"""Revudra: a decoder family without norms in front of its blocks -- every block reads the residual stream itself and only its
output is normed, x += m norm1(mixer(x)), x += m norm2(ff(x)) -- with a scaled embedding and scaled logits.  Its layers, in any
order given by config.json (``layers[i].type``), mix tokens by

* ``attention`` -- grouped-query attention through a sliding window, RMS norms over the whole query and the whole key projection,
  rotary positions on part of every head, a learned sink score per head, values mixed with those of the first mixing layer, a
  sigmoid gate per output element;
* ``lightning`` -- a matrix memory per head with a fixed decay, silu on queries, keys and values; one RMS norm over the
  concatenated heads, a sigmoid gate;
* ``latent_attention`` -- queries through one normed latent, keys and values of all heads through another, a rotated key part all
  heads share (neighbouring dimensions turn together), a learned sink per head, a sigmoid gate per head.

Feed-forward: dense with the square of relu, a mixture of silu-gated experts that the token id picks from a table, or none.

This module is the family's front: config.json -> ``SeqModelSpec``, checkpoint tensor names -> ``load_layer`` dicts, seeded
synthetic weights for benchmarks and tests.  The computation is models/seq_model.py + csrc/seq: the three mixers are the framework's
cached attention, retention and latent attention with their options, the router its routing by table.

config.json keys read here:
    architecture = "Revudra"; width; vocab; norm.eps; embedding.scale; residual_mult; logit_scale;
    layers[i].type = "attention": mixer.{heads, kv_heads, dim, vdim, scale, v_mix, mask: {size}, rot: {dims, base}}
    layers[i].type = "lightning": mixer.{heads, dim, vdim, decay: [heads numbers]}
    layers[i].type = "latent_attention": mixer.{heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot: {dims, base}}
    layers[i].mlp = null | {kind: "dense", ff} | {kind: "moe", router: {experts, top}, expert: {ff}}
Tensors (safetensors, [out, in]): embed, head, final.norm, and per layer ``l<i>.``: norm1, norm2, mix.{q, k, v, q.norm, k.norm, sink,
vmix, g, o}, mix.{q, k, v, norm, g, o}, mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, sink, g, o}, mlp.{up, down},
mlp.table and mlp.e<j>.{gate, up, down}.
"""
from __future__ import annotations

import json
import os

import torch

from .seq_model import SeqLayerSpec, SeqMlpSpec, SeqModelSpec, SeqStateModel

ARCHITECTURE = "Revudra"


def _rotary(l: SeqLayerSpec, rot: dict | None, most: int):
    if rot:
        l.rot_dims, l.rot_base = int(rot["dims"]), float(rot["base"])
        if l.rot_dims % 2 or l.rot_dims > most:
            raise ValueError("rot.dims must be even and no larger than the dimensions it turns")


def spec_from_config(cfg: dict) -> SeqModelSpec:
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: architecture = {cfg.get('architecture')!r}")
    mult = float(cfg.get("residual_mult", 1.0))
    layers, mixing = [], []
    for entry in cfg["layers"]:
        kind, mx = entry["type"], entry["mixer"]
        l = SeqLayerSpec(heads=int(mx["heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]), form="prenorm", pre_norm=False, post_norm=True,
                         residual_mult=mult, shift=False, depth_average=False)
        if kind == "attention":
            l.mixer, l.kv_heads, l.scale, l.window = "cached_attention", int(mx["kv_heads"]), float(mx["scale"]), int((mx.get("mask") or {}).get("size", 0))
            l.attn_mode, l.learned_sink, l.gate_kind, l.qk_norm_all = "softmax_sink", True, 2, True
            _rotary(l, mx.get("rot"), l.dim)
            if l.heads % l.kv_heads:
                raise ValueError("heads must be a multiple of kv_heads")
            if mx.get("v_mix"):
                mixing.append(l)
        elif kind == "lightning":
            l.mixer, l.decay, l.qkv_act, l.k_scale = "retention", [float(x) for x in mx["decay"]], "silu", 1.0
            l.out_norm, l.gate_act = True, "sigmoid"
            if len(l.decay) != l.heads:
                raise ValueError("decay: a number per head")
        elif kind == "latent_attention":
            l.mixer, l.rope_dim, l.kv_rank, l.q_rank, l.scale = kind, int(mx["rot_dim"]), int(mx["kv_rank"]), int(mx["q_rank"]), float(mx["scale"])
            l.window, l.attn_mode, l.learned_sink, l.gate_kind, l.rot_pairs = 0, "softmax_sink", True, 1, "neighbours"
            _rotary(l, mx.get("rot"), l.rope_dim)
        else:
            raise ValueError(f"unknown layer type '{kind}'")
        mlp = entry.get("mlp")
        if mlp is not None:
            mk = mlp.get("kind", "dense")
            if mk == "dense":
                l.mlp = SeqMlpSpec(shared_ff=int(mlp["ff"]), plain="relu2")
            elif mk == "moe":
                r = mlp["router"]
                l.mlp = SeqMlpSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), act="silu", route="table")
                if not 1 <= l.mlp.top <= l.mlp.experts:
                    raise ValueError("router: top must be between 1 and experts")
            else:
                raise ValueError(f"unknown feed-forward kind '{mk}'")
        layers.append(l)
    if len(mixing) > 1:                       # the first layer that mixes lends its values to the others
        mixing[0].v_mix = "source"
        for l in mixing[1:]:
            l.v_mix = "mix"
    eos = cfg.get("eos_token_id", [])
    return SeqModelSpec(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=layers, norm_groups=1, norm_eps=float(cfg["norm"]["eps"]),
                        embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), logit_scale=float(cfg.get("logit_scale", 1.0)),
                        eos_token_id=list(eos) if isinstance(eos, (list, tuple)) else [int(eos)])


def layer_tensor_names(spec: SeqModelSpec, i: int) -> dict:
    """load_layer key -> checkpoint tensor name(s) of layer i."""
    l, p = spec.layers[i], f"l{i}."
    m = p + "mix."
    names = {"post_norm": p + "norm1", "o": m + "o", "g": m + "g"}
    if l.mixer == "cached_attention":
        names.update({s: m + s for s in ("q", "k", "v", "sink")}, q_norm=m + "q.norm", k_norm=m + "k.norm")
        if l.v_mix == "mix":
            names["vmix"] = m + "vmix"
    elif l.mixer == "retention":
        names.update({s: m + s for s in ("q", "k", "v")}, out_norm=m + "norm")
    else:
        names.update({s: m + s for s in ("dq", "uq", "dkv", "uk", "uv", "sink")}, dq_norm=m + "dq.norm", dkv_norm=m + "dkv.norm")
    f = l.mlp
    if f is not None:
        names["post_norm2"] = p + "norm2"
        if f.experts:
            names["table"] = p + "mlp.table"
            names["experts"] = [tuple(f"{p}mlp.e{e}.{n}" for n in ("gate", "up", "down")) for e in range(f.experts)]
        else:
            names["dense"] = tuple(f"{p}mlp.{n}" for n in ("up", "down"))
    return names


class Revudra(SeqStateModel):
    """``Revudra(spec, ...)``; ``alloc()`` then ``load_checkpoint(path)`` or ``load_synthetic(seed)``."""

    def load_tensors(self, get):
        """``get(name) -> tensor`` for the family's tensor names."""
        read = lambda n: [read(x) for x in n] if isinstance(n, list) else tuple(get(x) for x in n) if isinstance(n, tuple) else get(n)
        self.load_head(get("embed"), get("head"), get("final.norm"))
        for i in range(self.num_layers):
            self.load_layer(i, {k: read(v) for k, v in layer_tensor_names(self.spec, i).items()})
        return self

    def load_checkpoint(self, path: str):
        from .checkpoint import SafetensorsIndex
        idx = SafetensorsIndex(path)
        self.load_tensors(idx.get)
        idx.close()
        self.weights_source = path
        return self

    def load_synthetic(self, seed: int = 1234, gen_device: str | None = None):
        """Seeded random weights of the architecture (benchmarks, tests)."""
        t = synth_tensors(self.spec, seed, gen_device or str(self.device))
        self.load_tensors(t.__getitem__)
        self.weights_source = f"synthetic(seed={seed})"
        return self


def synth_tensors(spec: SeqModelSpec, seed: int, dev="cpu") -> dict:
    """name -> bf16 (tables: int32) tensor, as a checkpoint would hold them, so that every dtype mode sees the same weights."""
    W, t = spec.width, {}
    gen = torch.Generator(device=dev).manual_seed(seed)
    r = lambda o, k, gain=1.0: (gain * k ** -0.5 * torch.randn(o, k, generator=gen, device=dev)).to(torch.bfloat16)
    vec = lambda n, s=1.0: (s * torch.randn(n, generator=gen, device=dev)).to(torch.bfloat16)
    one = lambda n, s=0.1: (1 + s * torch.randn(n, generator=gen, device=dev)).to(torch.bfloat16)
    t["embed"] = (torch.randn(spec.vocab, W, generator=gen, device=dev) / max(spec.embed_scale, 1e-6)).to(torch.bfloat16)
    t["head"], t["final.norm"] = r(spec.vocab, W), one(W)
    for i, l in enumerate(spec.layers):
        p = f"l{i}."
        m, hv, hd = p + "mix.", l.heads * l.vdim, l.heads * l.dim
        t[p + "norm1"], t[m + "o"] = one(W), r(W, hv)
        if l.mixer == "cached_attention":
            gd = l.kv_heads * l.dim
            t[m + "q"], t[m + "k"], t[m + "v"], t[m + "g"] = r(hd, W), r(gd, W), r(l.kv_heads * l.vdim, W), r(hv, W)
            t[m + "q.norm"], t[m + "k.norm"], t[m + "sink"] = one(hd), one(gd), vec(l.heads)
            if l.v_mix == "mix":
                t[m + "vmix"] = torch.tensor(0.3, device=dev).to(torch.bfloat16)
        elif l.mixer == "retention":
            t[m + "q"], t[m + "k"], t[m + "v"], t[m + "g"], t[m + "norm"] = r(hd, W), r(hd, W), r(hv, W), r(hv, W), one(hv)
        else:
            t[m + "dq"], t[m + "dq.norm"], t[m + "uq"] = r(l.q_rank, W), one(l.q_rank), r(l.heads * (l.dim + l.rope_dim), l.q_rank)
            t[m + "dkv"], t[m + "dkv.norm"] = r(l.kv_rank + l.rope_dim, W), one(l.kv_rank)
            t[m + "uk"], t[m + "uv"], t[m + "sink"], t[m + "g"] = r(hd, l.kv_rank), r(hv, l.kv_rank), vec(l.heads), r(l.heads, W)
        f = l.mlp
        if f is not None:
            t[p + "norm2"] = one(W)
            if f.experts:
                # every row of the table: `top` different experts
                t[p + "mlp.table"] = torch.rand(spec.vocab, f.experts, generator=gen, device=dev).argsort(-1)[:, :f.top].to(torch.int32)
                for e in range(f.experts):
                    t[f"{p}mlp.e{e}.gate"], t[f"{p}mlp.e{e}.up"], t[f"{p}mlp.e{e}.down"] = r(f.ff, W), r(f.ff, W), r(W, f.ff)
            else:
                t[p + "mlp.up"], t[p + "mlp.down"] = r(f.shared_ff, W), r(W, f.shared_ff)
    return t


def from_pretrained(path: str, device="cuda:0", dtype=torch.bfloat16, **kw) -> Revudra:
    """Model of a checkpoint directory (config.json + model.safetensors); ``alloc()`` loads the weights."""
    spec = spec_from_config(json.load(open(os.path.join(path, "config.json"))))
    model = Revudra(spec, device=device, dtype=dtype, model_name=path, **kw)
    base_alloc = model.alloc

    def alloc(**kwargs):
        base_alloc(**kwargs)
        if kwargs.get("synthetic") or "synthetic_seed" in kwargs:
            model.load_synthetic(kwargs.get("synthetic_seed", 1234))
        else:
            model.load_checkpoint(path)
        torch.cuda.synchronize(model.device)
        return model
    model.alloc = alloc
    return model
