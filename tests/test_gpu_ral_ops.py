"""Each mechanism the Ralapel family adds to the pre-norm step alone, on the GPU, against the plain statement in
oracle/ralapel.py: norms behind blocks, the embedding's norm, rows for the product in front of a pass, short convolutions
across steps, the gated delta rule and the state-space memory, the gated norms, latent attention whose neighbouring
dimensions turn together.  Inputs are shaped so that a fault shows: one key made dominant far back, a write that only the
delta rule takes off again, slots whose earlier owner left its numbers behind."""
import pytest
import torch

from oracle import ralapel as O

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def rnd(*shape, seed=0, scale=1.0):
    return scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def err(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def f32(t):
    return t.to(DEV, torch.float32).contiguous()


def as32(t):
    return t.float().double()


# ---------------------------------------------------------------------------------------------- norms
@pytest.mark.parametrize("n,width", [(7, 40), (5, 200), (3, 1100), (300, 256), (200, 2048), (2, 8192), (151, 4096), (4, 43)])
def test_norm_behind_a_block_residual_add_and_next_norm(n, width):
    from umbrella_b200 import ops_seq as K
    x, d = as32(rnd(n, width, seed=1, scale=2.0)), as32(rnd(n, width, seed=2, scale=30.0))
    pw, w = as32(rnd(width, seed=3, scale=0.3) + 1), as32(rnd(width, seed=4, scale=0.3) + 1)
    tot = x + O.rms_norm(d, pw, 1e-5)
    xs = f32(x)
    y, copy = K.add_post_norm(xs, f32(d), f32(pw), f32(w), 1e-5, want_copy=True)
    assert err(y, O.rms_norm(tot, w, 1e-5)) < 3e-6 and err(xs, tot) < 1e-6 and torch.equal(copy, xs)
    yb = K.add_post_norm(f32(x), f32(d), f32(pw), f32(w), 1e-5, dtype=torch.bfloat16)
    assert torch.equal(yb, y.to(torch.bfloat16))
    rows = torch.tensor([n - 1, 0, n - 1, n // 2], dtype=torch.int32, device=DEV)
    xs2 = f32(x)
    y2 = K.add_post_norm(xs2, f32(d), f32(pw), f32(w), 1e-5, rows=rows)
    assert err(y2, O.rms_norm(tot, w, 1e-5)[rows.cpu().long()]) < 3e-6 and torch.equal(xs2.cpu(), x.float())   # nothing written back


def test_a_silent_block_leaves_the_stream_finite():
    """A block output of zeros (or nearly) must meet eps inside the root, not a division by zero."""
    from umbrella_b200 import ops_seq as K
    for width in (64, 70):
        x, d = as32(rnd(3, width, seed=1)), torch.zeros(3, width, dtype=torch.float64)
        d[1] = as32(rnd(width, seed=2, scale=1e-3))
        w = torch.ones(width, dtype=torch.float64)
        xs = f32(x)
        K.add_post_norm(xs, f32(d), f32(w), f32(w), 1e-5)
        assert err(xs, x + O.rms_norm(d, w, 1e-5)) < 2e-6


@pytest.mark.parametrize("n,width", [(5, 40), (200, 256), (3, 51)])
def test_rows_of_a_pass(n, width):
    from umbrella_b200 import ops_seq as K
    x, d, pw = as32(rnd(n, width, seed=1)), as32(rnd(n, width, seed=2)), as32(rnd(width, seed=3) + 1)
    for dtype in (torch.float32, torch.bfloat16):
        for delta in (None, d):
            xs = f32(x)
            out = torch.full((n, 2 * width), 7.0, dtype=dtype, device=DEV)
            K.add_rows(xs, out, None if delta is None else f32(delta), f32(pw), 1e-6)
            tot = x if delta is None else x + O.rms_norm(d, pw, 1e-6)
            assert err(xs, tot) < 1e-6 and torch.equal(out[:, :width], xs.to(dtype)) and bool((out[:, width:] == 7.0).all())


def test_embedding_norm():
    from umbrella_b200 import ops_seq as K
    for width in (24, 300, 1024):
        for dtype in (torch.float32, torch.bfloat16):
            table = rnd(11, width, seed=1, scale=3.0).to(dtype)
            w = as32(rnd(width, seed=2, scale=0.3) + 1)
            ids = torch.tensor([3, 0, 10, 7, 7], dtype=torch.int32, device=DEV)
            copy = torch.zeros(5, 2 * width, dtype=dtype, device=DEV)
            y = K.embedding_norm(ids, table.to(DEV), f32(w), 1e-5, copy=copy[:, width:])
            assert err(y, O.rms_norm(table.double()[ids.cpu().long()], w, 1e-5)) < 2e-6
            assert torch.equal(copy[:, width:], y.to(dtype)) and float(copy[:, :width].abs().max()) == 0


# ---------------------------------------------------------------------------------------------- memories
SHAPES = [  # kind, heads, query/key heads (groups), dim (state), vdim, taps
    ("gated_delta", 4, 2, 12, 20, 4), ("gated_delta", 2, 2, 5, 7, 3), ("gated_delta", 6, 1, 64, 33, 2), ("gated_delta", 2, 1, 128, 40, 4),
    ("gated_delta", 1, 1, 200, 16, 4), ("gated_delta", 1, 1, 260, 9, 1), ("gated_delta", 40, 20, 16, 64, 4),
    ("ssd", 4, 2, 14, 10, 4), ("ssd", 3, 3, 33, 24, 1), ("ssd", 6, 2, 64, 32, 5), ("ssd", 2, 1, 128, 64, 4), ("ssd", 2, 1, 256, 17, 4),
    ("ssd", 1, 1, 500, 8, 3), ("ssd", 38, 19, 32, 64, 4)]


class MemoryCase:
    """One layer's memory with random constants, its projection rows, and the oracle's result for whole sequences."""

    def __init__(self, kind, heads, kv, dim, vdim, taps, slots=3, seed=0):
        self.kind, self.H, self.G, self.D, self.V, self.taps, self.slots = kind, heads, kv, dim, vdim, taps, slots
        gd, hv = kv * dim, heads * vdim
        self.ch = 2 * gd + hv
        self.cols = self.ch + hv + (2 if kind == "gated_delta" else 1) * heads
        self.conv_w, self.conv_b = as32(rnd(self.ch, taps, seed=seed + 1, scale=taps ** -0.5)), as32(rnd(self.ch, seed=seed + 2, scale=0.3))
        self.rate, self.bias = as32(rnd(heads, seed=seed + 3).exp()), as32(torch.linspace(0.0, -6.0, heads, dtype=torch.float64))
        self.skip = as32(rnd(heads, seed=seed + 4))
        self.parts = heads if kind == "gated_delta" else (2 if hv % 2 == 0 else 1)
        self.norm = as32(rnd(vdim if kind == "gated_delta" else hv, seed=seed + 5, scale=0.3) + 1)
        # every slot full of a former owner's numbers
        self.state = torch.full((slots, heads, vdim, dim), 5.0, device=DEV)
        self.conv_state = torch.full((2, slots, max(taps - 1, 1), self.ch), -3.0, device=DEV)
        from umbrella_b200 import ops_seq as K
        delta = kind == "gated_delta"
        self.keep = [f32(self.conv_w), None if delta else f32(self.conv_b), f32(self.rate), f32(self.bias), None if delta else f32(self.skip)]
        w, b, rate, bias, skip = self.keep
        self.mem, self.gate0 = K.memory_layout(kind, heads, kv, dim, vdim, taps, w, self.conv_state, rate, bias, self.state, b, skip)
        self.gpu_norm = f32(self.norm)

    def oracle(self, proj, eps=1e-5):
        n, H, G, D, V, gd, hv = proj.shape[0], self.H, self.G, self.D, self.V, self.G * self.D, self.H * self.V
        src = torch.tensor([a // (H // G) for a in range(H)])
        if self.kind == "gated_delta":
            y = O.silu(O.short_conv(proj[:, :self.ch], self.conv_w))
            q = O.unit_vector(y[:, :gd].reshape(n, G, D)) * D ** -0.5
            k = O.unit_vector(y[:, gd:2 * gd].reshape(n, G, D))
            gate, beta, a = proj[:, self.ch:self.ch + hv], torch.sigmoid(proj[:, self.ch + hv:self.ch + hv + H]), proj[:, self.ch + hv + H:]
            g = torch.exp(-self.rate * O.softplus(a + self.bias))
            o = O.delta_memory(q[:, src], k[:, src], y[:, 2 * gd:].reshape(n, H, V), beta, g)
            return (O.unit_rms(o, eps) * self.norm * O.silu(gate).reshape(n, H, V)).reshape(n, hv)
        z, y, dt = proj[:, :hv], O.silu(O.short_conv(proj[:, hv:hv + self.ch], self.conv_w, self.conv_b)), proj[:, hv + self.ch:]
        o = O.ssd_memory(y[:, :hv].reshape(n, H, V), y[:, hv:hv + gd].reshape(n, G, D)[:, src], y[:, hv + gd:].reshape(n, G, D)[:, src],
                         O.softplus(dt + self.bias), self.rate, self.skip).reshape(n, hv)
        return O.grouped_rms_norm(o * O.silu(z), self.norm, self.parts, eps)

    def step(self, rows, desc, eps=1e-5, dtype=torch.float32):
        from umbrella_b200 import ops_seq as K
        from umbrella_b200.ops_seq import RaggedBatch
        b, p = RaggedBatch(desc, DEV), f32(rows)
        qkv, gates, kq = K.memory_prep(p, self.mem, b, self.slots)
        o = K.memory_run(qkv, gates, kq, self.mem, b)
        return K.gated_norm(o, p[:, self.gate0:], self.parts, self.gpu_norm, self.kind == "ssd", eps, dtype)


def project(c, n, seed):
    """Projection rows in which one early token writes something that stands out, and a late one asks for it."""
    p = rnd(n, c.cols, seed=seed)
    p[:, -c.H:] -= 0.5
    p[min(5, n - 1)] *= 3.0
    p[n - 1, :c.ch] = p[min(5, n - 1), :c.ch]
    return as32(p)


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "-".join(str(x) for x in s))
def test_memories_whole_in_portions_and_token_by_token(shape):
    n = 70
    for schedule in ([n], [1] * n, [2, 30, 1, 1, 15, 21], [16, 16, 17, 15, 6], [3] * 23 + [1]):
        c = MemoryCase(*shape)
        proj = project(c, n, seed=9)
        out, pos, par = [], 0, 0
        for m in schedule:
            out.append(c.step(proj[pos:pos + m], [(1, m, pos, par)]))
            pos, par = pos + m, par ^ 1
        assert err(torch.cat(out), c.oracle(proj)) < 4e-5, schedule
        for slot in (0, 2):                                     # nobody else's state was touched
            assert bool((c.state[slot] == 5.0).all()) and bool((c.conv_state[:, slot] == -3.0).all())


@pytest.mark.parametrize("shape", [SHAPES[0], SHAPES[3], SHAPES[6], SHAPES[7], SHAPES[10], SHAPES[13]], ids=lambda s: "-".join(str(x) for x in s))
def test_memories_of_a_ragged_batch(shape):
    """Sequences of unequal length out of non-adjacent slots, over two steps: first a long one, then a mixture of a later
    portion, a decoded token and a fresh sequence in a slot that another sequence has just used."""
    c = MemoryCase(*shape, slots=6)
    lens = {4: 150, 1: 1, 3: 130, 0: 2}
    seqs = {s: project(c, n + 40, seed=50 + s) for s, n in lens.items()}
    out = c.step(torch.cat([seqs[s][:n] for s, n in lens.items()]), [(s, n, 0, 0) for s, n in lens.items()])
    o = 0
    for s, n in lens.items():
        assert err(out[o:o + n], c.oracle(seqs[s])[:n]) < 4e-5, s
        o += n
    fresh = project(c, 11, seed=77)
    out = c.step(torch.cat([seqs[4][150:151], fresh, seqs[1][1:31]]), [(4, 1, 150, 1), (3, 11, 0, 1), (1, 30, 1, 1)])
    assert err(out[:1], c.oracle(seqs[4])[150:151]) < 4e-5
    assert err(out[1:12], c.oracle(fresh)) < 4e-5
    assert err(out[12:], c.oracle(seqs[1])[1:31]) < 4e-5


def test_the_delta_rule_takes_off_what_the_memory_returns():
    """The same unit key written twice with strength 1 and no decay: the second value replaces the first instead of adding
    to it (and an orthogonal key is left alone) -- which a plain additive memory would get wrong by the whole first value."""
    from umbrella_b200 import _lib_seq as S, ops_seq as K
    from umbrella_b200.ops_seq import RaggedBatch
    D, V = 16, 24
    state = torch.zeros(1, 1, V, D, device=DEV)
    e = torch.eye(D, dtype=torch.float64)
    v = as32(rnd(3, V, seed=1))
    q, k = torch.stack([e[0], e[0], e[1]]), torch.stack([e[0], e[0], e[1]])
    qkv = f32(torch.cat([q, k, v], dim=1))
    gates = f32(torch.tensor([[[0.0, 1.0]]] * 3))
    for rule, second in ((S.UMBS_MEMORY_DELTA, v[1]), (S.UMBS_MEMORY_ADD, v[0] + v[1])):
        state.zero_()
        mem = S.Memory()
        mem.rule, mem.heads, mem.kv_heads, mem.dim, mem.vdim, mem.taps = rule, 1, 1, D, V, 1
        mem.off_q, mem.off_k, mem.off_v, mem.state = 0, D, 2 * D, state.data_ptr()
        o = K.memory_run(qkv, gates, f32((q * k).sum(-1, keepdim=True)), mem, RaggedBatch([(0, 3, 0, 0)], DEV))
        assert err(o, torch.stack([v[0], second, v[2]])) < 1e-6
        assert err(state[0, 0, :, 0], second) < 1e-6 and err(state[0, 0, :, 1], v[2]) < 1e-6


def test_a_memory_without_decay_keeps_its_first_token():
    """Slow heads carry the first token over a thousand steps of decoding: compared at the end, against a sequence whose first
    token differs."""
    c = MemoryCase("ssd", 2, 1, 32, 16, 4)
    c.rate = as32(torch.tensor([1e-4, 1e-3]))
    c.keep[2].copy_(f32(c.rate))
    n = 600
    proj = project(c, n, seed=3) * 0.5
    other = proj.clone()
    other[0] *= -40.0
    ref, alt = c.oracle(proj), c.oracle(other)
    assert err(ref[-1], alt[-1]) > 1e-3
    for p, r in ((proj, ref), (other, alt)):
        c.step(p[:300], [(1, 300, 0, 0)])
        out = [c.step(p[i:i + 1], [(1, 1, i, (i - 299) & 1)]) for i in range(300, n)]
        assert err(torch.cat(out), r[300:]) < 4e-5


@pytest.mark.parametrize("n,width,parts,w_len", [(5, 40, 5, 40), (9, 96, 4, 24), (3, 2048, 1, 2048), (3, 2046, 2, 2046), (200, 1024, 8, 128), (2, 6000, 3, 6000)])
def test_gated_norms(n, width, parts, w_len):
    """Gate in front of the norm and behind it; parts of a warp and of a block; a weight shared by the parts."""
    from umbrella_b200 import ops_seq as K
    o, z, w = as32(rnd(n, width, seed=1, scale=3.0)), as32(rnd(n, width + 3, seed=2)), as32(rnd(w_len, seed=3) + 1)
    g = O.silu(z[:, :width])
    full = w.repeat(width // w_len)
    first, behind = O.grouped_rms_norm(o * g, full, parts, 1e-5), O.grouped_rms_norm(o, full, parts, 1e-5) * g
    for zz in (f32(z), f32(z[:, :width])):                      # a gate whose rows are no multiple of a piece, and one whose are
        assert err(K.gated_norm(f32(o), zz, parts, f32(w), True, 1e-5), first) < 4e-6
        assert err(K.gated_norm(f32(o), zz, parts, f32(w), False, 1e-5), behind) < 4e-6
        assert err(K.gated_norm(f32(o), zz, parts, f32(w), False, 1e-5, torch.bfloat16), behind) < 1e-2


# ---------------------------------------------------------------------------------------------- latent attention, neighbours turn together
@pytest.mark.parametrize("H,D,R,V,rank", [(3, 10, 6, 14, 20), (2, 16, 8, 24, 36), (1, 32, 64, 48, 64), (2, 200, 4, 150, 24)])
@pytest.mark.parametrize("part", ["unrotated", "rotated"])
def test_latent_attention_with_neighbouring_pairs(H, D, R, V, rank, part):
    """A one-layer model whose far key stands out for a late query, by its unrotated or its rotated part: whole, in portions,
    token by token; and the pairing itself (turning i with i + R / 2 instead gives other numbers)."""
    import ral_helpers as U
    cfg = U.model(48, 60, [U.latent(H, D, R, V, rank, base=100.0)])
    t = U.random_tensors(cfg, seed=H + D)
    n, far = 140, 2
    seq = torch.randint(0, 5, (n,), generator=torch.Generator().manual_seed(1)).tolist()
    seq[far], seq[n - 1] = 55, 56                               # tokens that occur once: what answers, what asks
    d, scale = {k: v.double() for k, v in t.items()}, cfg["layers"][0]["mixer"]["scale"]
    h = O.rms_norm(O.rms_norm(d["embed"], d["embed.norm"], 1e-5), d["l0.norm1"], 1e-5)
    if part == "unrotated":                # head 0's query of token 56: a score of 14 with token 55's key, 0 with the others'
        c = O.rms_norm((h[[55, 56, 0, 1, 2, 3, 4]] @ d["l0.mix.dkv"].T)[:, :rank], d["l0.mix.dkv.norm"], 1e-5)
        want = torch.linalg.pinv(c @ d["l0.mix.uk"][:D].T)[:, 0] * 14.0 / scale
        rows = slice(0, D)
    else:                                  # ... or with its shared part (a long one), turned back by the distance
        d["l0.mix.dkv"][rank:] += torch.outer(rnd(R, seed=5, scale=6.0), h[55]) / float(h[55] @ h[55])
        t["l0.mix.dkv"] = d["l0.mix.dkv"].to(torch.bfloat16).float()
        want = O.rotate_pairs((t["l0.mix.dkv"].double()[rank:] @ h[55])[None], 100.0, first=far - (n - 1))[0]
        want = want * (14.0 / scale / float(want @ want))
        rows = slice(D, D + R)
    d["l0.mix.q"][rows] += torch.outer(want - d["l0.mix.q"][rows] @ h[56], h[56]) / float(h[56] @ h[56])
    t["l0.mix.q"] = d["l0.mix.q"].to(torch.bfloat16).float()
    om, pm = U.oracle_model(cfg, t), U.product_model(cfg, t, torch.float32)
    ref = O.forward(om, seq)[0]
    gone = list(seq)
    gone[far] = 58
    assert U.row_err(O.forward(om, gone)[0][-1:], ref[-1:]) > 0.03          # the far key decides the last row
    if R > 2:
        halves = dict(t)
        order = torch.cat([torch.arange(0, R, 2), torch.arange(1, R, 2)])
        both = t["l0.mix.dkv"].clone(), t["l0.mix.q"].reshape(H, D + R, -1).clone()
        both[0][rank:], both[1][:, D:] = both[0][rank:][order], both[1][:, D:][:, order]
        halves["l0.mix.dkv"], halves["l0.mix.q"] = both[0], both[1].reshape(t["l0.mix.q"].shape)
        assert U.row_err(O.forward(U.oracle_model(cfg, halves), seq)[0], ref) > 1e-2
    for pieces in ([n], [100] + [1] * 40, [2, 61, 1, 1, 64, 11], [7] * 20):
        slot, out, i = pm.cache.alloc_slot(), [], 0
        for m in pieces:
            out.append(pm.forward([(slot, seq[i:i + m], range(m))]))
            i += m
        pm.cache.free_slot(slot)
        assert U.row_err(torch.cat(out), ref) < 3e-5, pieces


def test_neighbour_pairs_reordered_as_halves():
    from umbrella_b200.models.seq_model import pair_rows_as_halves
    w = torch.arange(12.0)[:, None]
    assert pair_rows_as_halves(w, 3, 6).flatten().tolist() == [0, 1, 2, 3, 5, 7, 4, 6, 8, 9, 10, 11]
    assert pair_rows_as_halves(w.reshape(2, 6, 1), 2, 4).flatten().tolist() == [0, 1, 2, 4, 3, 5, 6, 7, 8, 10, 9, 11]
