"""Ralapel: a decoder family with a norm in front of and behind every block (x += norm1b(mixer(norm1(x))), then
x += norm2b(ff(norm2(x)))), a norm on the embedding, and a span of layers that runs several times with the same weights --
in front of every pass x <- W [x; x0] brings the embedding output back in, and every pass keeps caches and states of its own.
Its layers, in any order given by config.json (``layers[i].type``), mix tokens by

* ``latent_attention`` -- direct queries, keys and values of all heads from one RMS-normed low-rank latent per token, a rotated
  key part all heads share (neighbouring dimensions turn together), ordinary causal softmax;
* ``delta`` -- the gated delta rule: short convolution + silu on q, k and v, unit q and k, one decay and one write strength
  per head and token, a matrix memory whose write first takes off what the memory already returns for the key; unit RMS
  per head, a weight heads share, a silu gate;
* ``mamba2`` -- a state-space memory: one projection for gate, input, input and read-out vectors (shared by groups of heads)
  and step sizes, short convolution with bias + silu, decay from the step size, a skip per head; silu gate, then an RMS norm
  in equal parts.

Feed-forward: dense gelu-gated (tanh form) or none.

This module is the family's front: config.json -> ``SeqModelSpec``, checkpoint tensor names -> ``load_layer`` dicts, seeded
synthetic weights for benchmarks and tests.  The computation is models/seq_model.py + csrc/seq: the attention is the
framework's latent-attention mixer with direct queries, the two recurrent kinds its rank-one memories.

config.json keys read here:
    architecture = "Ralapel"; width; vocab; norm.eps; loop = null | {start, stop, times};
    layers[i].type = "latent_attention": mixer.{heads, dim, rot_dim, vdim, kv_rank, scale, rot: {dims, base}}
    layers[i].type = "delta": mixer.{heads, kv_heads, dim, vdim, conv}
    layers[i].type = "mamba2": mixer.{heads, vdim, state, groups, norm_groups, conv}
    layers[i].mlp = null | {kind: "dense", ff}
Tensors (safetensors, [out, in]): embed, embed.norm, loop.in, head, final.norm, and per layer ``l<i>.``: norm1, norm1b, norm2,
norm2b, mix.{q, dkv, dkv.norm, uk, uv, o}, mix.{q, k, v (+ .conv), b, a, A_log, dt_bias, norm, g, o},
mix.{in, conv, conv.b, dt_bias, A_log, D, norm, o}, mlp.{gate, up, down}.
"""
from __future__ import annotations

import json
import os

import torch

from .seq_model import SeqLayerSpec, SeqMlpSpec, SeqModelSpec, SeqStateModel

ARCHITECTURE = "Ralapel"


def spec_from_config(cfg: dict) -> SeqModelSpec:
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: architecture = {cfg.get('architecture')!r}")
    layers = []
    for entry in cfg["layers"]:
        kind, mx = entry["type"], entry["mixer"]
        l = SeqLayerSpec(heads=int(mx["heads"]), vdim=int(mx["vdim"]), form="prenorm", post_norm=True, shift=False, depth_average=False)
        if kind == "latent_attention":
            l.mixer, l.dim, l.rope_dim, l.kv_rank, l.scale = kind, int(mx["dim"]), int(mx["rot_dim"]), int(mx["kv_rank"]), float(mx["scale"])
            l.q_rank, l.window, l.attn_mode, l.gate_kind = 0, 0, "softmax", 0
            l.rot_dims, l.rot_base, l.rot_pairs = int(mx["rot"]["dims"]), float(mx["rot"]["base"]), "neighbours"
            if l.rot_dims % 2 or l.rot_dims > l.rope_dim:
                raise ValueError("rot.dims must be even and at most rot_dim")
        elif kind in ("delta", "mamba2"):
            l.taps = int(mx["conv"])
            if kind == "delta":
                l.mixer, l.dim, l.kv_heads = "gated_delta", int(mx["dim"]), int(mx["kv_heads"])
            else:
                l.mixer, l.dim, l.kv_heads, l.norm_parts = "ssd", int(mx["state"]), int(mx["groups"]), int(mx["norm_groups"])
                if l.heads * l.vdim % l.norm_parts:
                    raise ValueError("norm_groups must divide heads * vdim")
            if l.heads % l.kv_heads or l.taps < 1:
                raise ValueError("heads must be a multiple of the query / key heads (groups), conv at least one tap")
        else:
            raise ValueError(f"unknown layer type '{kind}'")
        mlp = entry.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind '{mlp['kind']}'")
            l.mlp = SeqMlpSpec(shared_ff=int(mlp["ff"]), act="gelu_tanh")
        layers.append(l)
    loop, eos = cfg.get("loop"), cfg.get("eos_token_id", [])
    return SeqModelSpec(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=layers, norm_groups=1, norm_eps=float(cfg["norm"]["eps"]),
                        embed_norm=True, loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None,
                        eos_token_id=list(eos) if isinstance(eos, (list, tuple)) else [int(eos)])


def layer_tensor_names(spec: SeqModelSpec, i: int) -> dict:
    """load_layer key -> checkpoint tensor name(s) of layer i."""
    l, p = spec.layers[i], f"l{i}."
    m = p + "mix."
    names = {"norm": p + "norm1", "post_norm": p + "norm1b", "o": m + "o"}
    if l.mixer == "latent_attention":
        names.update({s: m + s for s in ("q", "dkv", "uk", "uv")}, dkv_norm=m + "dkv.norm")
    elif l.mixer == "gated_delta":
        names.update({s: m + s for s in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "g")}, out_norm=m + "norm",
                     **{s + "_conv": f"{m}{s}.conv" for s in "qkv"})
    else:
        names.update({s: m + s for s in ("in", "conv", "dt_bias", "A_log", "D")}, conv_b=m + "conv.b", out_norm=m + "norm")
    if l.mlp is not None:
        names.update(norm2=p + "norm2", post_norm2=p + "norm2b", dense=tuple(f"{p}mlp.{n}" for n in ("gate", "up", "down")))
    return names


class Ralapel(SeqStateModel):
    """``Ralapel(spec, ...)``; ``alloc()`` then ``load_checkpoint(path)`` or ``load_synthetic(seed)``."""

    def load_tensors(self, get):
        """``get(name) -> tensor`` for the family's tensor names."""
        self.load_head(get("embed"), get("head"), get("final.norm"), embed_norm=get("embed.norm"),
                       loop_in=get("loop.in") if self.spec.loop is not None else None)
        for i in range(self.num_layers):
            self.load_layer(i, {k: tuple(get(n) for n in v) if isinstance(v, tuple) else get(v)
                                for k, v in layer_tensor_names(self.spec, i).items()})
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
    """name -> bf16 tensor (as a checkpoint would hold them), so that every dtype mode sees the same weights."""
    W, t = spec.width, {}
    gen = torch.Generator(device=dev).manual_seed(seed)
    r = lambda o, k, gain=1.0: (gain * k ** -0.5 * torch.randn(o, k, generator=gen, device=dev)).to(torch.bfloat16)
    vec = lambda n, s=0.1: (s * torch.randn(n, generator=gen, device=dev)).to(torch.bfloat16)
    one = lambda n, s=0.1: (1 + s * torch.randn(n, generator=gen, device=dev)).to(torch.bfloat16)
    t["embed"], t["embed.norm"], t["head"], t["final.norm"] = r(spec.vocab, W), one(W), r(spec.vocab, W), one(W)
    if spec.loop is not None:
        t["loop.in"] = r(W, 2 * W)
    for i, l in enumerate(spec.layers):
        p = f"l{i}."
        m, hv, gd = p + "mix.", l.heads * l.vdim, l.kv_heads * l.dim
        t[p + "norm1"], t[p + "norm1b"], t[m + "o"] = one(W), one(W), r(W, hv)
        if l.mixer == "latent_attention":
            t[m + "q"], t[m + "dkv"] = r(l.heads * (l.dim + l.rope_dim), W, 2.0), r(l.kv_rank + l.rope_dim, W, 2.0)
            t[m + "dkv.norm"], t[m + "uk"], t[m + "uv"] = one(l.kv_rank), r(l.heads * l.dim, l.kv_rank, 2.0), r(hv, l.kv_rank)
        else:
            t[m + "A_log"], t[m + "dt_bias"] = vec(l.heads, 0.5), vec(l.heads, 0.5) - 2.0
            if l.mixer == "gated_delta":
                for s, n in (("q", gd), ("k", gd), ("v", hv)):
                    t[m + s], t[f"{m}{s}.conv"] = r(n, W), r(n, l.taps)
                t[m + "b"], t[m + "a"], t[m + "g"], t[m + "norm"] = r(l.heads, W), r(l.heads, W), r(hv, W), one(l.vdim)
            else:
                t[m + "in"], t[m + "conv"], t[m + "conv.b"] = r(2 * hv + 2 * gd + l.heads, W), r(hv + 2 * gd, l.taps), vec(hv + 2 * gd)
                t[m + "D"], t[m + "norm"] = one(l.heads), one(hv)
        if l.mlp is not None:
            ff = l.mlp.shared_ff
            t[p + "norm2"], t[p + "norm2b"] = one(W), one(W)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = r(ff, W), r(ff, W), r(W, ff)
    return t


def from_pretrained(path: str, device="cuda:0", dtype=torch.bfloat16, **kw) -> Ralapel:
    """Model of a checkpoint directory (config.json + model.safetensors); ``alloc()`` loads the weights."""
    spec = spec_from_config(json.load(open(os.path.join(path, "config.json"))))
    model = Ralapel(spec, device=device, dtype=dtype, model_name=path, **kw)
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
