"""Test-only helpers for the Ralapel family: small random models, built twice from the same tensors -- as the oracle's plain
dict (float64, oracle/ralapel.py) and as the product model (a checkpoint directory read by the family's config reader and
loader).  A configuration here is the family's config.json itself."""
import json
import os

import torch


def latent(heads, dim, rot_dim, vdim, kv_rank, base=300.0, scale=None, ff=0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale or 1.4 * (dim + rot_dim) ** -0.5,
             rot=dict(base=base, dims=rot_dim))
    return dict(type="latent_attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None)


def delta(heads, kv_heads, dim, vdim, conv=4, ff=0):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
                mlp=dict(kind="dense", ff=ff) if ff else None)


def mamba2(heads, vdim, state, groups=1, norm_groups=1, conv=4, ff=0):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv),
                mlp=dict(kind="dense", ff=ff) if ff else None)


def model(width, vocab, layers, loop=None, eps=1e-5):
    return dict(architecture="Ralapel", width=width, vocab=vocab, norm=dict(eps=eps), layers=layers,
                loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)


# every branch: the three kinds in and around a loop that runs three times, with and without feed-forward; heads = query / key
# heads and several per one; one group and several, one norm part and several; taps 4, 3, 2 and 1; sizes no vector load takes
MIXED = model(72, 101, [
    delta(6, 3, 12, 20, conv=3, ff=40),
    mamba2(4, 10, 14, groups=2, norm_groups=5, conv=4),
    latent(3, 10, 6, 14, 20),
    mamba2(2, 24, 33, groups=1, norm_groups=1, conv=1, ff=52),
    latent(2, 8, 12, 20, 28, base=1000.0, ff=36),
    delta(2, 2, 11, 7, conv=2),
], loop=(1, 4, 3))
# dimensions the vectorised kernels and the bf16 tensor-core product take
ALIGNED = model(128, 160, [
    mamba2(4, 64, 64, groups=2, norm_groups=2, ff=192),
    delta(4, 2, 64, 32, ff=128),
    latent(4, 32, 32, 64, 64, base=1e4, ff=256),
], loop=(0, 2, 2), eps=1e-6)
# sizes no tensor-core tile takes, shallow enough for bf16 rounding to stay small
ODD = model(72, 90, [delta(4, 2, 12, 20, conv=3), mamba2(4, 10, 14, groups=2, norm_groups=5), latent(3, 10, 6, 14, 20, ff=44)])
# no loop at all
PLAIN = model(64, 77, [delta(4, 1, 16, 24), latent(2, 16, 8, 12, 16, ff=48), mamba2(6, 8, 20, groups=3, norm_groups=2)])


def _bf(t):
    return t.to(torch.bfloat16).to(torch.float32)          # values a bf16 checkpoint can hold


def random_tensors(cfg, seed=0):
    """name -> fp32 tensor (bf16-representable), with the family's checkpoint names.  The decays of a layer's heads spread from
    memories of a few tokens to memories that outlast every test, so that a lost state shows."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    r = lambda o, k, gain=1.0: _bf(gain * k ** -0.5 * torch.randn(o, k, generator=g))
    vec = lambda n, s=0.2: _bf(s * torch.randn(n, generator=g))
    one = lambda n, s=0.2: _bf(1 + s * torch.randn(n, generator=g))
    t = {"embed": _bf(torch.randn(cfg["vocab"], W, generator=g)), "embed.norm": one(W), "final.norm": one(W), "head": r(cfg["vocab"], W)}
    if cfg.get("loop"):
        t["loop.in"] = r(W, 2 * W)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q, H, V = p + "mix.", m["heads"], m["vdim"]
        t[p + "norm1"], t[p + "norm1b"], t[q + "o"] = one(W), one(W), r(W, H * V)
        if L["type"] == "latent_attention":
            t[q + "q"], t[q + "dkv"], t[q + "dkv.norm"] = r(H * (m["dim"] + m["rot_dim"]), W, 1.3), r(m["kv_rank"] + m["rot_dim"], W, 1.3), one(m["kv_rank"])
            t[q + "uk"], t[q + "uv"] = r(H * m["dim"], m["kv_rank"], 1.3), r(H * V, m["kv_rank"])
        else:
            t[q + "A_log"] = _bf(torch.linspace(-1.0, 1.0, H) + 0.1 * torch.randn(H, generator=g))
            t[q + "dt_bias"] = _bf(torch.linspace(0.0, -5.0, H)[torch.randperm(H, generator=g)])
            if L["type"] == "delta":
                for s, n in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", H * V)):
                    t[q + s], t[f"{q}{s}.conv"] = r(n, W, 1.5), r(n, m["conv"], 1.5)
                # queries that resemble their keys: a token's read-out then seldom cancels to nothing in front of the unit norm, which
                # would magnify rounding by any factor
                t[q + "q"], t[q + "q.conv"] = _bf(t[q + "k"] + 0.5 * t[q + "q"]), _bf(t[q + "k.conv"] + 0.3 * t[q + "q.conv"])
                t[q + "b"], t[q + "a"], t[q + "g"], t[q + "norm"] = r(H, W), r(H, W), r(H * V, W, 1.5), one(V)
            else:
                gn = m["groups"] * m["state"]
                t[q + "in"], t[q + "conv"], t[q + "conv.b"] = r(2 * H * V + 2 * gn + H, W, 1.5), r(H * V + 2 * gn, m["conv"], 1.5), vec(H * V + 2 * gn)
                t[q + "D"], t[q + "norm"] = one(H), one(H * V)
        f = L["mlp"]
        if f is not None:
            t[p + "norm2"], t[p + "norm2b"] = one(W), one(W)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = r(f["ff"], W, 1.5), r(f["ff"], W), r(W, f["ff"])
    return t


def oracle_model(cfg, t):
    from oracle import ralapel as O
    return O.from_tensors(cfg, t)


def write_checkpoint(path, cfg, t):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    json.dump(cfg, open(os.path.join(path, "config.json"), "w"))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}, os.path.join(path, "model.safetensors"))
    return path


def product_model(cfg, t, dtype=torch.float32, device="cuda:0", slots=4, tmp=None, **kw):
    """The product model over the same tensors, through the registry, the family's config reader and its loader."""
    import tempfile
    from umbrella_b200.models.auto_model import AutoModelLM
    d = write_checkpoint(tmp or tempfile.mkdtemp(prefix="ralckpt"), cfg, t)
    m = AutoModelLM.from_pretrained(d, device=device, dtype=dtype, slots=slots, **kw)
    m.alloc()
    return m


def row_errs(a, b):
    """Per-row rms difference relative to the rms of the whole reference."""
    a, b = a.double().cpu(), b.double().cpu()
    return (a - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt().clamp_min(1e-30)


def row_err(a, b):
    return float(row_errs(a, b).max())


def close(a, b, worst=1.5e-3, typical=1e-4):
    """fp32 product against float64 oracle.  A deep random stack magnifies rounding at single rows (where a unit norm meets an
    output that nearly cancels: the plain statement in fp32 strays as far), so both the worst and the median row are bounded;
    a lost state, key or tap moves rows by 1e-2 and more."""
    e = row_errs(a, b)
    return float(e.max()) < worst and float(e.median()) < typical
