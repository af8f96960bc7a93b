"""Test-only helpers for the Revudra family: small random models, built twice from the same tensors -- as the oracle's plain
dict (float64, oracle/revudra.py) and as the product model (a checkpoint directory read by the family's config reader and
loader).  A configuration here is the family's config.json itself."""
import json
import os

import torch


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))


def attention(heads, kv_heads, dim, vdim, window, rot_dims, base=300.0, scale=None, v_mix=True, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window), scale=scale or 1.4 * dim ** -0.5, v_mix=v_mix,
             rot=dict(dims=rot_dims, base=base))
    return dict(type="attention", mixer=m, mlp=mlp)


def lightning(heads, dim, vdim, decay=None, mlp=None):
    """Decays spread from a memory of a few tokens to one that outlasts every test, so that a lost state shows."""
    decay = decay or [1.0 - 2.0 ** (-1.0 - 10.0 * h / heads) for h in range(heads)]
    return dict(type="lightning", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay), mlp=mlp)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=100.0, scale=None, mlp=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale or 1.4 * (dim + rot_dim) ** -0.5,
             rot=dict(base=base, dims=rot_dim))
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def model(width, vocab, layers, eps=1e-5, embed=3.0, mult=0.6, logit=0.4):
    return dict(architecture="Revudra", width=width, vocab=vocab, norm=dict(eps=eps), embedding=dict(scale=embed), residual_mult=mult,
                logit_scale=logit, layers=layers)


# every branch: the mixing source is not the first layer and not the first attention layer; windows, bases, head counts and scales of
# their own; values wider and narrower than keys; dense, routed (one, two and three experts per token) and no feed-forward; sizes no
# vector load takes
MIXED = model(72, 101, [
    lightning(5, 11, 14, mlp=moe(5, 3, 20)),
    attention(4, 2, 12, 20, 9, 8, v_mix=False),
    attention(6, 3, 10, 14, 17, 10, base=50.0, mlp=dense(44)),
    latent(3, 10, 6, 14, 26, 20, mlp=moe(3, 1, 28)),
    attention(3, 3, 16, 14, 24, 4, base=1e4, mlp=moe(6, 2, 12)),
    lightning(2, 20, 9),
    attention(8, 1, 6, 42, 1, 2, mlp=dense(30)),
    latent(2, 8, 12, 20, 17, 28, base=1000.0),
])
# dimensions the vectorised kernels and the bf16 tensor-core product take; windows longer than a key tile
ALIGNED = model(128, 160, [
    attention(4, 2, 32, 64, 80, 16, base=1e4, mlp=dense(192)),
    lightning(4, 64, 32, mlp=moe(8, 2, 64)),
    latent(4, 32, 32, 64, 96, 64, base=1e4, mlp=moe(4, 2, 96)),
    attention(8, 4, 64, 32, 33, 64, mlp=moe(8, 4, 32)),
], eps=1e-6, embed=8.0, mult=0.8, logit=0.2)
# sizes no tensor-core tile takes, shallow enough for bf16 rounding to stay small
ODD = model(72, 90, [attention(4, 2, 12, 20, 19, 6, mlp=dense(44)), lightning(4, 10, 14), latent(3, 10, 6, 14, 26, 20, mlp=moe(5, 2, 20))])


def _bf(t):
    return t.to(torch.bfloat16).to(torch.float32)          # values a bf16 checkpoint can hold


def random_tensors(cfg, seed=0):
    """name -> fp32 tensor (bf16-representable; tables int32), with the family's checkpoint names."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    r = lambda o, k, gain=1.0: _bf(gain * k ** -0.5 * torch.randn(o, k, generator=g))
    one = lambda n, s=0.2: _bf(1 + s * torch.randn(n, generator=g))
    t = {"embed": _bf(torch.randn(V, W, generator=g) / cfg["embedding"]["scale"]), "final.norm": one(W), "head": r(V, W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q, H, Vd, D = p + "mix.", m["heads"], m["vdim"], m["dim"]
        t[p + "norm1"], t[q + "o"] = one(W), r(W, H * Vd)
        if L["type"] == "attention":
            G = m["kv_heads"]
            t[q + "q"], t[q + "k"], t[q + "v"], t[q + "g"] = r(H * D, W), r(G * D, W), r(G * Vd, W), r(H * Vd, W, 1.5)
            t[q + "q.norm"], t[q + "k.norm"] = one(H * D), one(G * D)
            t[q + "sink"] = _bf(torch.randn(H, generator=g))
            if m["v_mix"]:
                t[q + "vmix"] = _bf(0.2 + 0.6 * torch.rand((), generator=g))
        elif L["type"] == "lightning":
            t[q + "k"], t[q + "v"], t[q + "g"], t[q + "norm"] = r(H * D, W, 1.5), r(H * Vd, W, 1.5), r(H * Vd, W, 1.5), one(H * Vd)
            # queries that resemble their keys: a token's read-out then seldom cancels to nothing in front of the norm, which would
            # magnify rounding by any factor
            t[q + "q"] = _bf(t[q + "k"] + 0.5 * r(H * D, W, 1.5))
        else:
            R, T = m["kv_rank"], m["rot_dim"]
            t[q + "dq"], t[q + "dq.norm"], t[q + "uq"] = r(m["q_rank"], W), one(m["q_rank"]), r(H * (D + T), m["q_rank"], 1.3)
            t[q + "dkv"], t[q + "dkv.norm"] = r(R + T, W), one(R)
            t[q + "uk"], t[q + "uv"], t[q + "g"] = r(H * D, R, 1.3), r(H * Vd, R), r(H, W, 1.5)
            t[q + "sink"] = _bf(torch.randn(H, generator=g))
        f = L["mlp"]
        if f is not None:
            t[p + "norm2"] = one(W)
            if f["kind"] == "dense":
                t[p + "mlp.up"], t[p + "mlp.down"] = r(f["ff"], W), r(W, f["ff"])
            else:
                E, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
                t[p + "mlp.table"] = torch.rand(V, E, generator=g).argsort(-1)[:, :top].to(torch.int32)
                for e in range(E):
                    for n, o, k in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                        t[f"{p}mlp.e{e}.{n}"] = r(o, k)
    return t


def oracle_model(cfg, t):
    from oracle import revudra as O
    return O.from_tensors(cfg, t)


def write_checkpoint(path, cfg, t):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    json.dump(cfg, open(os.path.join(path, "config.json"), "w"))
    save_file({k: (v if v.dtype == torch.int32 else v.to(torch.bfloat16)).contiguous() for k, v in t.items()}, os.path.join(path, "model.safetensors"))
    return path


def product_model(cfg, t, dtype=torch.float32, device="cuda:0", slots=4, tmp=None, **kw):
    """The product model over the same tensors, through the registry, the family's config reader and its loader."""
    import tempfile
    from umbrella_b200.models.auto_model import AutoModelLM
    d = write_checkpoint(tmp or tempfile.mkdtemp(prefix="revckpt"), cfg, t)
    m = AutoModelLM.from_pretrained(d, device=device, dtype=dtype, slots=slots, **kw)
    m.alloc()
    return m


def row_errs(a, b):
    """Per-row rms difference relative to the rms of the whole reference."""
    a, b = a.double().cpu(), b.double().cpu()
    return (a - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt().clamp_min(1e-30)


def row_err(a, b):
    return float(row_errs(a, b).max())


def close(a, b, worst=1e-3, typical=5e-5):
    """fp32 product against float64 oracle.  Both the worst and the median row are bounded: a norm behind a block whose output
    nearly cancels magnifies rounding at single rows (the plain statement in fp32 strays as far); a lost state, key or expert moves
    rows by 1e-2 and more."""
    e = row_errs(a, b)
    return float(e.max()) < worst and float(e.median()) < typical
