"""Plain, slow statement of the Ralapel mechanisms, one function per mechanism, in float64 on the CPU, written from the
equations -- the oracle the CUDA path is tested against.  It shares no code with umbrella_b200.  A model is

    {"eps", "embed", "embed_norm", "loop": None | {"start", "stop", "times", "w"}, "layers": [...], "final_norm", "head"}
    layer: {"type": "latent_attention" | "delta" | "mamba2", "norm1", "norm1b", "norm2", "norm2b", "mix": {...},
            "mlp": None | {gate, up, down}}          (norm2, norm2b absent without a feed-forward)
      latent_attention mix: {heads, dim, rot_dim, vdim, kv_rank, scale, base, q, dkv, dkv_norm, uk, uv, o}
      delta mix:  {heads, kv_heads, dim, vdim, q, k, v, q_conv, k_conv, v_conv, b, a, A_log, dt_bias, norm, g, o}
      mamba2 mix: {heads, vdim, state, groups, norm_groups, in, conv, conv_b, dt_bias, A_log, D, norm, o}

Every function takes a whole sequence [n, .]: no cache, no state, no batching.  Position i of a result depends on
tokens 0..i of that one sequence, which is what the product must reproduce however it is fed.
"""
import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------------------------------------- element-wise pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def short_conv(u, w, bias=None):
    """Causal convolution over time, per channel: y[t, c] = bias[c] + sum_j w[c, j] u[t - (taps - 1) + j, c], zeros in front."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u) if bias is None else bias.expand_as(u).clone()
    for t in range(n):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def rotate_pairs(x, base, first=0):
    """x [n, ..., d]: neighbours (2i, 2i + 1) turn by (first + row) base^(-2i / d)."""
    d = x.shape[-1]
    out = x.clone()
    for r in range(x.shape[0]):
        for i in range(d // 2):
            a = (first + r) * base ** (-2.0 * i / d)
            u, v = x[r, ..., 2 * i], x[r, ..., 2 * i + 1]
            out[r, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[r, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


# ---------------------------------------------------------------------------------------------- mixers
def causal_softmax(s):
    n = s.shape[-1]
    s = s.masked_fill(~torch.tril(torch.ones(n, n, dtype=torch.bool)), -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_attention(h, m, eps):
    """Keys and values of all heads from one normed latent per token; a rotated key part all heads share."""
    n, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ m["q"].T).reshape(n, H, D + R)
    low = h @ m["dkv"].T
    c = rms_norm(low[:, :m["kv_rank"]], m["dkv_norm"], eps)
    shared = rotate_pairs(low[:, m["kv_rank"]:], m["base"])
    turned = rotate_pairs(q[:, :, D:], m["base"])
    k = (c @ m["uk"].T).reshape(n, H, D)
    v = (c @ m["uv"].T).reshape(n, H, V)
    out = torch.zeros(n, H, V, dtype=F64)
    for a in range(H):
        s = (q[:, a, :D] @ k[:, a].T + turned[:, a] @ shared.T) * m["scale"]
        out[:, a] = causal_softmax(s) @ v[:, a]
    return out.reshape(n, H * V) @ m["o"].T


def delta_memory(q, k, v, beta, g):
    """Per head: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  q, k [n, H, D]; v [n, H, V]; beta, g [n, H]."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def delta_inputs(h, m):
    """q, k (unit vectors, q times dim^-1/2; spread over the value heads), v, beta, g of the gated delta rule."""
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_vector(silu(short_conv(h @ m["q"].T, m["q_conv"])).reshape(n, G, D)) * D ** -0.5
    k = unit_vector(silu(short_conv(h @ m["k"].T, m["k_conv"])).reshape(n, G, D))
    v = silu(short_conv(h @ m["v"].T, m["v_conv"])).reshape(n, H, V)
    beta = torch.sigmoid(h @ m["b"].T)
    g = torch.exp(-torch.exp(m["A_log"]) * softplus(h @ m["a"].T + m["dt_bias"]))
    src = torch.tensor([a // (H // G) for a in range(H)])
    return q[:, src], k[:, src], v, beta, g


def delta(h, m, eps):
    n, H, V = h.shape[0], m["heads"], m["vdim"]
    o = delta_memory(*delta_inputs(h, m))
    o = unit_rms(o, eps) * m["norm"] * silu(h @ m["g"].T).reshape(n, H, V)
    return o.reshape(n, H * V) @ m["o"].T


def ssd_memory(x, B, C, dt, A, D):
    """Per head: S <- exp(-A dt) S + dt B x^T; y = S^T C + D x.  x [n, H, V]; B, C [n, H, N]; dt [n, H]; A, D [H]."""
    n, H, V = x.shape
    S = torch.zeros(H, B.shape[2], V, dtype=F64)
    out = torch.zeros(n, H, V, dtype=F64)
    for t in range(n):
        S = torch.exp(-A * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, C[t]) + D[:, None] * x[t]
    return out


def grouped_rms_norm(y, w, groups, eps):
    n, width = y.shape
    return unit_rms(y.reshape(n, groups, width // groups), eps).reshape(n, width) * w


def mamba2(h, m, eps):
    n, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    p = h @ m["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, m["conv"], m["conv_b"]))
    x = xbc[:, :inner].reshape(n, H, V)
    src = torch.tensor([a // (H // G) for a in range(H)])
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)[:, src]
    C = xbc[:, inner + G * N:].reshape(n, G, N)[:, src]
    y = ssd_memory(x, B, C, softplus(dt + m["dt_bias"]), torch.exp(m["A_log"]), m["D"]).reshape(n, inner)
    return grouped_rms_norm(y * silu(z), m["norm"], m["norm_groups"], eps) @ m["o"].T


# ---------------------------------------------------------------------------------------------- feed-forward, model
def feed_forward(h, m):
    return (gelu_tanh(h @ m["gate"].T) * (h @ m["up"].T)) @ m["down"].T


MIXERS = {"latent_attention": latent_attention, "delta": delta, "mamba2": mamba2}


def schedule(n_layers, loop):
    """[(layer, first of a pass)] in the order the layers run."""
    if loop is None:
        return [(i, False) for i in range(n_layers)]
    body = range(loop["start"], loop["stop"])
    return [(i, False) for i in range(loop["start"])] + [(i, i == loop["start"]) for _ in range(loop["times"]) for i in body] + \
        [(i, False) for i in range(loop["stop"], n_layers)]


def forward(model, tokens):
    """-> (logits [n, vocab], residual stream after every layer run [runs, n, width]) of one sequence, float64."""
    eps = model["eps"]
    x = x0 = rms_norm(model["embed"][torch.tensor(tokens)], model["embed_norm"], eps)
    streams = []
    for i, entry in schedule(len(model["layers"]), model["loop"]):
        L = model["layers"][i]
        if entry:
            x = torch.cat([x, x0], dim=-1) @ model["loop"]["w"].T
        x = x + rms_norm(MIXERS[L["type"]](rms_norm(x, L["norm1"], eps), L["mix"], eps), L["norm1b"], eps)
        if L["mlp"] is not None:
            x = x + rms_norm(feed_forward(rms_norm(x, L["norm2"], eps), L["mlp"]), L["norm2b"], eps)
        streams.append(x)
    return rms_norm(x, model["final_norm"], eps) @ model["head"].T, torch.stack(streams)


def from_tensors(cfg, t):
    """config dict (as config.json holds it) + name -> tensor  ->  the model dict above, float64."""
    f = lambda name: t[name].to(F64)
    layers = []
    for i, e in enumerate(cfg["layers"]):
        p, c = f"l{i}.", e["mixer"]
        if e["type"] == "latent_attention":
            assert c["rot"]["dims"] == c["rot_dim"]
            mix = dict(heads=c["heads"], dim=c["dim"], rot_dim=c["rot_dim"], vdim=c["vdim"], kv_rank=c["kv_rank"], scale=c["scale"],
                       base=c["rot"]["base"], dkv_norm=f(p + "mix.dkv.norm"), **{s: f(p + "mix." + s) for s in ("q", "dkv", "uk", "uv", "o")})
        elif e["type"] == "delta":
            mix = dict(heads=c["heads"], kv_heads=c["kv_heads"], dim=c["dim"], vdim=c["vdim"],
                       **{s + "_conv": f(f"{p}mix.{s}.conv") for s in "qkv"},
                       **{s: f(p + "mix." + s) for s in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "g", "o")})
        else:
            mix = dict(heads=c["heads"], vdim=c["vdim"], state=c["state"], groups=c["groups"], norm_groups=c["norm_groups"],
                       conv_b=f(p + "mix.conv.b"), **{s: f(p + "mix." + s) for s in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")})
        layer = dict(type=e["type"], norm1=f(p + "norm1"), norm1b=f(p + "norm1b"), mix=mix, mlp=None)
        if e.get("mlp") is not None:
            layer.update(norm2=f(p + "norm2"), norm2b=f(p + "norm2b"), mlp={s: f(p + "mlp." + s) for s in ("gate", "up", "down")})
        layers.append(layer)
    loop = cfg.get("loop")
    return dict(eps=cfg["norm"]["eps"], embed=f("embed"), embed_norm=f("embed.norm"), layers=layers, final_norm=f("final.norm"),
                head=f("head"), loop=None if loop is None else dict(loop, w=f("loop.in")))
