"""Plain, slow statement of the Revudra mechanisms, one function per mechanism, in float64 on the CPU, written from the
equations -- the oracle the CUDA path is tested against.  It shares no code with umbrella_b200.  A model is

    {"eps", "mult", "embed_scale", "logit_scale", "embed", "layers": [...], "final_norm", "head"}
    layer: {"type": "attention" | "lightning" | "latent_attention", "norm1", "norm2", "mix": {...}, "mlp": None | {...}}
      attention mix: {heads, kv_heads, dim, vdim, window, scale, base, rot_dims, v_mix, q, k, v, q_norm, k_norm, sink, vmix, g, o}
      lightning mix: {heads, dim, vdim, decay [heads], q, k, v, norm, g, o}
      latent_attention mix: {heads, dim, rot_dim, vdim, kv_rank, scale, base, dq, dq_norm, uq, dkv, dkv_norm, uk, uv, sink, g, o}
      dense mlp: {up, down};  mixture: {experts: [(gate, up, down), ...], table [vocab, top]}

Every function takes a whole sequence [n, .]: no cache, no state, no batching.  Position i of a result depends on
tokens 0..i of that one sequence, which is what the product must reproduce however it is fed.
"""
import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------------------------------------- element-wise pieces
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def rotate_halves(x, dims, base, first=0):
    """x [n, ..., d]: dimensions i and i + dims / 2 of the first ``dims`` turn by (first + row) base^(-2i / dims)."""
    out, half = x.clone(), dims // 2
    for r in range(x.shape[0]):
        for i in range(half):
            a = (first + r) * base ** (-2.0 * i / dims)
            u, v = x[r, ..., i], x[r, ..., i + half]
            out[r, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[r, ..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def rotate_pairs(x, base, first=0):
    """x [n, ..., d]: neighbours (2i, 2i + 1) turn by (first + row) base^(-2i / d)."""
    d, out = x.shape[-1], x.clone()
    for r in range(x.shape[0]):
        for i in range(d // 2):
            a = (first + r) * base ** (-2.0 * i / d)
            u, v = x[r, ..., 2 * i], x[r, ..., 2 * i + 1]
            out[r, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[r, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def visible(n, window):
    """[n, n] bool: the last ``window`` keys up to the row itself (window 0: all of them)."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & ((d < window) if window else torch.ones_like(d, dtype=torch.bool))


def sink_softmax(s, mask, sink):
    """Weights of one head's scores s [n, n] with exp(sink) in the denominator beside the visible keys."""
    s = s.masked_fill(~mask, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


# ---------------------------------------------------------------------------------------------- mixers
def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention(h, m, eps, first_values):
    """-> (output, the layer's unmixed values): grouped-query attention through a window, norms over all query (key) rows at
    once, sink, values mixed with those of the first mixing layer, gate per output element."""
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ m["q"].T, m["q_norm"], eps).reshape(n, H, D)
    k = rms_norm(h @ m["k"].T, m["k_norm"], eps).reshape(n, G, D)
    v = h @ m["v"].T
    own = v
    if m["v_mix"] and first_values is not None:
        v = mix_values(v, first_values, m["vmix"])
    q, k, v = rotate_halves(q, m["rot_dims"], m["base"]), rotate_halves(k, m["rot_dims"], m["base"]), v.reshape(n, G, V)
    mask = visible(n, m["window"])
    out = torch.zeros(n, H, V, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = sink_softmax(q[:, a] @ k[:, g].T * m["scale"], mask, m["sink"][a]) @ v[:, g]
    return (out.reshape(n, H * V) * torch.sigmoid(h @ m["g"].T)) @ m["o"].T, own


def decayed_memory(q, k, v, decay):
    """Per head: S <- decay S + k v^T; o = S^T q.  q, k [n, H, D]; v [n, H, V]; decay [H]."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for t in range(n):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def lightning(h, m, eps):
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ m[s].T).reshape(n, H, -1) for s in "qkv")
    o = decayed_memory(q, k, v, torch.tensor(m["decay"], dtype=F64)).reshape(n, H * V)
    return (rms_norm(o, m["norm"], eps) * torch.sigmoid(h @ m["g"].T)) @ m["o"].T


def latent_attention(h, m, eps):
    """Queries from one normed latent, keys and values of all heads from another; a rotated key part all heads share; sink; a
    gate per head."""
    n, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (rms_norm(h @ m["dq"].T, m["dq_norm"], eps) @ m["uq"].T).reshape(n, H, D + R)
    low = h @ m["dkv"].T
    c = rms_norm(low[:, :m["kv_rank"]], m["dkv_norm"], eps)
    shared = rotate_pairs(low[:, m["kv_rank"]:], m["base"])
    turned = rotate_pairs(q[:, :, D:], m["base"])
    k = (c @ m["uk"].T).reshape(n, H, D)
    v = (c @ m["uv"].T).reshape(n, H, V)
    gate = torch.sigmoid(h @ m["g"].T)
    mask = visible(n, 0)
    out = torch.zeros(n, H, V, dtype=F64)
    for a in range(H):
        s = (q[:, a, :D] @ k[:, a].T + turned[:, a] @ shared.T) * m["scale"]
        out[:, a] = sink_softmax(s, mask, m["sink"][a]) @ v[:, a] * gate[:, a:a + 1]
    return out.reshape(n, H * V) @ m["o"].T


# ---------------------------------------------------------------------------------------------- feed-forward, model
def dense(x, m):
    return relu_squared(x @ m["up"].T) @ m["down"].T


def mixture(x, m, tokens):
    """The token id alone picks its experts; each weighs 1 / top."""
    out = torch.zeros_like(x)
    top = m["table"].shape[1]
    for t, tok in enumerate(tokens):
        for e in m["table"][tok].tolist():
            gate, up, down = m["experts"][e]
            out[t] += ((silu(x[t] @ gate.T) * (x[t] @ up.T)) @ down.T) / top
    return out


def forward(model, tokens):
    """-> (logits [n, vocab], residual stream after every layer [layers, n, width]) of one sequence, float64."""
    eps, mult = model["eps"], model["mult"]
    x = model["embed"][torch.tensor(tokens)] * model["embed_scale"]
    streams, first = [], None
    for L in model["layers"]:
        if L["type"] == "attention":
            y, own = attention(x, L["mix"], eps, first)
            if L["mix"]["v_mix"] and first is None:
                first = own
        else:
            y = (lightning if L["type"] == "lightning" else latent_attention)(x, L["mix"], eps)
        x = x + mult * rms_norm(y, L["norm1"], eps)
        if L["mlp"] is not None:
            y = mixture(x, L["mlp"], tokens) if "table" in L["mlp"] else dense(x, L["mlp"])
            x = x + mult * rms_norm(y, L["norm2"], eps)
        streams.append(x)
    return rms_norm(x, model["final_norm"], eps) @ model["head"].T * model["logit_scale"], torch.stack(streams)


def from_tensors(cfg, t):
    """config dict (as config.json holds it) + name -> tensor  ->  the model dict above, float64."""
    f = lambda name: t[name].to(F64)
    layers = []
    for i, e in enumerate(cfg["layers"]):
        p, c = f"l{i}.", e["mixer"]
        q = p + "mix."
        if e["type"] == "attention":
            mix = dict(heads=c["heads"], kv_heads=c["kv_heads"], dim=c["dim"], vdim=c["vdim"], window=c["mask"]["size"], scale=c["scale"],
                       base=c["rot"]["base"], rot_dims=c["rot"]["dims"], v_mix=bool(c.get("v_mix")), q_norm=f(q + "q.norm"),
                       k_norm=f(q + "k.norm"), vmix=f(q + "vmix") if c.get("v_mix") else None,
                       **{s: f(q + s) for s in ("q", "k", "v", "sink", "g", "o")})
        elif e["type"] == "lightning":
            mix = dict(heads=c["heads"], dim=c["dim"], vdim=c["vdim"], decay=c["decay"], **{s: f(q + s) for s in ("q", "k", "v", "norm", "g", "o")})
        else:
            assert c["rot"]["dims"] == c["rot_dim"]
            mix = dict(heads=c["heads"], dim=c["dim"], rot_dim=c["rot_dim"], vdim=c["vdim"], kv_rank=c["kv_rank"], scale=c["scale"],
                       base=c["rot"]["base"], dq_norm=f(q + "dq.norm"), dkv_norm=f(q + "dkv.norm"),
                       **{s: f(q + s) for s in ("dq", "uq", "dkv", "uk", "uv", "sink", "g", "o")})
        layer = dict(type=e["type"], norm1=f(p + "norm1"), mix=mix, mlp=None)
        if e.get("mlp") is not None:
            layer["norm2"] = f(p + "norm2")
            if e["mlp"]["kind"] == "dense":
                layer["mlp"] = dict(up=f(p + "mlp.up"), down=f(p + "mlp.down"))
            else:
                layer["mlp"] = dict(table=t[p + "mlp.table"].long(), experts=[tuple(f(f"{p}mlp.e{j}.{n}") for n in ("gate", "up", "down"))
                                                                             for j in range(e["mlp"]["router"]["experts"])])
        layers.append(layer)
    return dict(eps=cfg["norm"]["eps"], mult=cfg["residual_mult"], embed_scale=cfg["embedding"]["scale"], logit_scale=cfg["logit_scale"],
                embed=f("embed"), layers=layers, final_norm=f("final.norm"), head=f("head"))
