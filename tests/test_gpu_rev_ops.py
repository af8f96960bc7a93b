"""The mechanisms Revudra adds, each kernel alone on the GPU against the plain oracle (oracle/revudra.py): decayed memories with one
norm over the heads, attention preparation with norms over whole rows and mixed values, sinks and windows decided by one
standing-out key, latents and per-head gates, activations of a product's first columns, routing by token id, norms behind blocks
with a multiplier."""
import pytest
import torch

from oracle import revudra as O
from rev_helpers import row_err

pytestmark = pytest.mark.gpu
DEV, F64 = "cuda:0", torch.float64


def rnd(*shape, seed=0, scale=1.0):
    return scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def Q():
    from umbrella_b200 import ops_seq
    return ops_seq


def S():
    from umbrella_b200 import _lib_seq
    return _lib_seq


def turn_freq(dims, base):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32, device=DEV) if dims else torch.zeros(1, device=DEV)


# ---------------------------------------------------------------------------------------------- lightning memories
def lightning_ref(rows, H, D, V, decay, w, eps, parts=1):
    rows = rows.to(F64)
    q, k, v, g = rows.split([H * D, H * D, H * V, H * V], dim=1)
    n = rows.shape[0]
    o = O.decayed_memory(q.reshape(n, H, D), k.reshape(n, H, D), v.reshape(n, H, V), decay.to(F64)).reshape(n, parts, -1)
    o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)).reshape(n, H * V)
    return o * w.to(F64) * torch.sigmoid(g)


SHAPES = [(1, 8, 8), (3, 5, 7), (2, 32, 32), (4, 33, 50), (2, 64, 128), (5, 100, 36), (2, 128, 128), (1, 200, 64), (1, 512, 40)]


@pytest.mark.parametrize("H,D,V", SHAPES)
def test_lightning_whole_portions_and_ragged(H, D, V):
    n, eps = 150, 1e-5
    decay = torch.tensor([1.0 - 2.0 ** (-1 - 9.0 * h / H) for h in range(H)], dtype=torch.float32)
    w, rows = 1 + 0.2 * rnd(H * V, seed=3), rnd(n, 2 * H * (D + V), seed=D)
    ref = lightning_ref(rows, H, D, V, decay, w, eps)
    state = torch.full((4, H, D, V), 1e6, device=DEV)             # slots full of a former owner's numbers
    f, d, wd, r = turn_freq(0, 1.0), decay.to(DEV), w.to(DEV), rows.to(DEV)
    opts = dict(k_scale=1.0, norm_w=wd, gate_act=S().UMBS_GATE_SIGMOID)

    def feed(sizes, slot, segments=True):
        out, p = [], 0
        for m in sizes:
            b = Q().RaggedBatch([(slot, m, p, 0)], DEV)
            out.append(Q().retention(r[p:p + m].contiguous(), b, H, D, V, 0, f, d, eps, state, segments=segments, **opts))
            p += m
        return torch.cat(out)
    for slot, sizes, seg in ((0, [n], True), (1, [n], False), (2, [1] * n, True), (3, [2, 2, 16, 1, 17, 112], True), (0, [15, 130, 2, 3], True)):
        assert row_err(feed(sizes, slot, seg), ref) < 2e-4, (sizes[:4], seg)
    # unequal sequences in one step, out of non-adjacent slots, over two steps
    lens, slots = [(40, 1), (1, 60), (23, 23)], [3, 0, 2]
    at = [0, 41, 102]
    for part in (0, 1):
        pos = [0 if part == 0 else a for a, _ in lens]
        take = [l[part] for l in lens]
        idx = torch.cat([torch.arange(a + p, a + p + t) for a, p, t in zip(at, pos, take)])
        b = Q().RaggedBatch([(s, t, p, 0) for s, t, p in zip(slots, take, pos)], DEV)
        got = Q().retention(r[idx.to(DEV)].contiguous(), b, H, D, V, 0, f, d, eps, state, **opts)
        o = 0
        for a, p, t in zip(at, pos, take):
            alone = lightning_ref(rows[a:a + p + t], H, D, V, decay, w, eps)[p:]
            assert row_err(got[o:o + t], alone) < 2e-4
            o += t


def test_lightning_carries_a_first_token_far():
    """A first token written large decides the last read-out 700 tokens later; with a slower decay for one head than the other."""
    H, D, V, n = 2, 16, 24, 700
    decay = torch.tensor([0.9995, 0.98])
    rows = rnd(n, 2 * H * (D + V), seed=5)
    rows[0, H * D:2 * H * D] *= 60.0
    rows[-1, :H * D] = rows[0, H * D:2 * H * D] / 60.0
    w = torch.ones(H * V)
    ref = lightning_ref(rows, H, D, V, decay, w, 1e-6)
    lost = lightning_ref(rows[1:], H, D, V, decay, w, 1e-6)
    assert row_err(lost[-1:], ref[-1:]) > 0.1
    state, r = torch.zeros(1, H, D, V, device=DEV), rows.to(DEV)
    for sizes in ([n], [350, 349, 1], [690] + [1] * 10):
        out, p = [], 0
        for m in sizes:
            out.append(Q().retention(r[p:p + m].contiguous(), Q().RaggedBatch([(0, m, p, 0)], DEV), H, D, V, 0, turn_freq(0, 1.0), decay.to(DEV), 1e-6,
                                     state, k_scale=1.0, norm_w=w.to(DEV), gate_act=S().UMBS_GATE_SIGMOID))
            p += m
        assert row_err(torch.cat(out)[-1:], ref[-1:]) < 2e-4


@pytest.mark.parametrize("parts", [1, 2, 6])
@pytest.mark.parametrize("n,width", [(1, 36), (9, 90), (5, 768), (3, 3072)])
def test_gated_norm_with_a_sigmoid(n, width, parts):
    o, g, w = rnd(n, width, seed=1, scale=3.0), rnd(n, width + 5, seed=2, scale=2.0), 1 + 0.3 * rnd(width, seed=3)
    u = o.to(F64).reshape(n, parts, -1)
    ref = (u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-5)).reshape(n, width) * w.to(F64) * torch.sigmoid(g[:, :width].to(F64))
    got = Q().gated_norm(o.to(DEV), g.to(DEV)[:, :width], parts, w.to(DEV), False, 1e-5, gate_act=S().UMBS_GATE_SIGMOID)
    assert row_err(got, ref) < 2e-6


# ---------------------------------------------------------------------------------------------- attention preparation
@pytest.mark.parametrize("H,G,D,V,rot", [(1, 1, 4, 4, 4), (3, 1, 10, 7, 6), (4, 2, 32, 64, 16), (8, 4, 64, 32, 64), (2, 2, 20, 12, 0), (16, 4, 128, 128, 64)])
@pytest.mark.parametrize("n", [1, 5, 80])
def test_attention_prep_norms_whole_rows_and_mixes_values(H, G, D, V, rot, n):
    base, eps, lam, p0 = 500.0, 1e-5, 0.37, 11
    ld = (H + G) * D + G * V + H * V
    # heads of very different size: a norm per head would give other numbers
    proj = rnd(n, ld, seed=H) * torch.cat([torch.repeat_interleave(torch.arange(1, H + G + 1).float(), D), torch.ones(G * V + H * V)])
    qw, kw, first = 1 + 0.3 * rnd(H * D, seed=4), 1 + 0.3 * rnd(G * D, seed=5), rnd(n, G * V, seed=6)
    x = proj.to(F64)
    q = O.rotate_halves(O.rms_norm(x[:, :H * D], qw.to(F64), eps).reshape(n, H, D), rot, base, p0).reshape(n, -1)
    k = O.rotate_halves(O.rms_norm(x[:, H * D:(H + G) * D], kw.to(F64), eps).reshape(n, G, D), rot, base, p0).reshape(n, -1)
    v = x[:, (H + G) * D:(H + G) * D + G * V]
    b = Q().RaggedBatch([(0, n, p0, 0)], DEV)
    P = proj.to(DEV)
    args = (b, H, G, D, V, rot, turn_freq(rot, base), qw.to(DEV), kw.to(DEV), eps)
    src = torch.zeros(n, G * V, device=DEV)
    for mode, store, vals in ((S().UMBS_VMIX_NONE, None, v), (S().UMBS_VMIX_SOURCE, src, v), (S().UMBS_VMIX_MIX, first.to(DEV), O.mix_values(v, first.to(F64), lam))):
        gq, gkv = Q().attention_prep_rows(P, *args, v_mix=mode, v_lambda=lam, v_source=store)
        assert row_err(gq, q) < 5e-6 and row_err(gkv[:, :G * D], k) < 5e-6 and row_err(gkv[:, G * D:], vals) < 1e-6
    assert torch.equal(src.cpu(), proj[:, (H + G) * D:(H + G) * D + G * V])


# ---------------------------------------------------------------------------------------------- sinks and windows
def attention_ref(q, k, v, window, scale, sink, gate):
    """q [n, H, D], k [n, G, D], v [n, G, V], float64 -> [n, H V]."""
    n, H, _ = q.shape
    rep, mask = H // k.shape[1], O.visible(n, window)
    out = [O.sink_softmax(q[:, a] @ k[:, a // rep].T * scale, mask, sink[a]) @ v[:, a // rep] for a in range(H)]
    return torch.stack(out, 1).reshape(n, -1) * torch.sigmoid(gate)


@pytest.mark.parametrize("H,G,D,V,window", [(4, 2, 16, 20, 9), (3, 1, 40, 12, 64), (2, 2, 128, 128, 65), (6, 3, 10, 70, 200), (2, 1, 32, 32, 1), (4, 1, 64, 64, 0)])
def test_windowed_attention_with_sinks(H, G, D, V, window):
    """One key stands out among all others: rows just inside and just outside its window, in prompts, portions and decoding; a sink
    that takes nearly everything, one that takes nothing, and one in between."""
    n, scale = 230, 0.7 * D ** -0.5
    q, k, v, gate = rnd(n, H, D, seed=1), rnd(n, G, D, seed=2), rnd(n, G, V, seed=3), rnd(n, H * V, seed=4)
    far = 20
    u = torch.nn.functional.normalize(rnd(D, seed=5), dim=0)
    k[far] = 3.0 * u * D ** 0.5
    reach = window if window else 150
    for i in {far, far + 1, far + reach - 1, far + reach, far + reach + 1, n - 1}:
        if i < n:
            q[i] = 3.0 * u * D ** 0.5
    sink = torch.tensor([6.0, -8.0, 0.5, 2.0, -1.0, 1.0])[:H]
    ref = attention_ref(q.to(F64), k.to(F64), v.to(F64), window, scale, sink.to(F64), gate.to(F64))
    if window > 1 and far + window < n:               # the key must show at the last row that sees it, and only there
        v2 = v.clone()
        v2[far] += 1.0
        moved = (attention_ref(q.to(F64), k.to(F64), v2.to(F64), window, scale, sink.to(F64), gate.to(F64)) - ref).abs().amax(-1)
        assert moved[far + window - 1] > 1e-2 and moved[far + window] == 0.0
    QD, KV, GD = q.reshape(n, -1).to(DEV), torch.cat([k.reshape(n, -1), v.reshape(n, -1)], 1).to(DEV), gate.to(DEV)
    kvl = window if window else 256
    for dt, tol in ((torch.float32, 3e-5), (torch.bfloat16, 3e-2)):
        for sizes in ([n], [far + reach if far + reach < n else 200] + [1] * 30, [2, 2, 64, 1, 63, 2, 40, 56], [1] * 90):
            cache, out, p = torch.full((3, kvl, KV.shape[1]), 99.0, device=DEV, dtype=dt), [], 0
            for m in sizes:
                m = min(m, n - p)
                if m <= 0:
                    break
                b = Q().RaggedBatch([(1, m, p, 0)], DEV)
                out.append(Q().cached_attention(QD[p:p + m].to(dt).contiguous(), KV[p:p + m].to(dt).contiguous(), cache, b, H, G, D, V, scale,
                                                mode=S().UMBS_ATTN_SOFTMAX_SINK, window=window, sink=sink.to(DEV), gate=GD[p:p + m]))
                p += m
            assert row_err(torch.cat(out), ref[:p]) < tol, (dt, sizes[:3])


def test_sink_of_a_split_decode_step():
    """Long contexts spread a decoded row over several blocks: the sink counts once, not once per block."""
    H, G, D, V, n = 2, 1, 32, 32, 1500
    q, k, v = rnd(1, H, D, seed=1), rnd(n, G, D, seed=2), rnd(n, G, V, seed=3)
    sink, gate = torch.tensor([7.0, -3.0]), rnd(1, H * V, seed=4)
    s = torch.einsum("hd,ngd->hn", q[0].to(F64), k.to(F64)) * 0.2
    e, es = torch.exp(s), torch.exp(sink.to(F64))
    ref = ((e / (e.sum(-1, keepdim=True) + es[:, None])) @ v[:, 0].to(F64)).reshape(1, -1) * torch.sigmoid(gate.to(F64))
    kv = torch.cat([k.reshape(n, -1), v.reshape(n, -1)], 1).to(DEV)
    cache = torch.zeros(1, n, kv.shape[1], device=DEV)
    cache[0, :n - 1] = kv[:-1]
    b = Q().RaggedBatch([(0, 1, n - 1, 0)], DEV)
    for split in (True, False):
        got = Q().cached_attention(q.reshape(1, -1).to(DEV), kv[-1:].contiguous(), cache, b, H, G, D, V, 0.2, mode=S().UMBS_ATTN_SOFTMAX_SINK,
                                   sink=sink.to(DEV), gate=gate.to(DEV), split=split, append=False)
        assert row_err(got, ref) < 2e-5


# ---------------------------------------------------------------------------------------------- latents
@pytest.mark.parametrize("H,D,T,R,QR", [(2, 8, 6, 20, 17), (3, 10, 12, 28, 26), (4, 32, 32, 64, 96), (16, 128, 64, 512, 768)])
def test_latent_preparation_in_two_pieces(H, D, T, R, QR):
    n, eps, base, p0 = 37, 1e-5, 200.0, 5
    f = turn_freq(T, base)
    low, qs = rnd(n, QR + R + T + H, seed=1), rnd(n, H * (D + T), seed=2)
    qn, kn = 1 + 0.2 * rnd(QR, seed=3), 1 + 0.2 * rnd(R, seed=4)
    b = Q().RaggedBatch([(0, n, p0, 0)], DEV)
    cq, c = Q().latent_low_prep(low.to(DEV), b, QR, qn.to(DEV), R, kn.to(DEV), T, T, f, eps)
    x = low.to(F64)
    # halves here: the loader reorders the rows of neighbour pairs
    shared = O.rotate_halves(x[:, QR + R:QR + R + T], T, base, p0)
    assert row_err(cq, O.rms_norm(x[:, :QR], qn.to(F64), eps)) < 3e-6
    assert row_err(c, torch.cat([O.rms_norm(x[:, QR:QR + R], kn.to(F64), eps), shared], 1)) < 3e-6
    q, q_abs = Q().latent_query_turn(qs.to(DEV), b, H, D, T, R, T, f)
    y = qs.to(F64).reshape(n, H, D + T).clone()
    y[:, :, D:] = O.rotate_halves(y[:, :, D:], T, base, p0)
    assert row_err(q, y.reshape(n, -1)) < 3e-6
    assert row_err(q_abs[:, :, R:].reshape(n, -1), y[:, :, D:].reshape(n, -1)) < 3e-6 and float(q_abs[:, :, :R].abs().max()) == 0.0


@pytest.mark.parametrize("M", [1, 3, 9, 40, 150])
@pytest.mark.parametrize("H,V,R", [(3, 14, 20), (4, 64, 64), (2, 32, 96)])
def test_gate_per_head(M, H, V, R):
    """The per-head gate behind the value product (every kernel of the product) and behind attention over per-head keys."""
    o, w, gate = rnd(M, H * R, seed=1), rnd(H, V, R, seed=2, scale=R ** -0.5), rnd(M, H + 3, seed=3, scale=2.0)
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 1e-2)):
        a, b = o.to(dt), w.to(dt)
        ref = torch.einsum("mhr,hvr->mhv", a.to(F64).reshape(M, H, R), b.to(F64)) * torch.sigmoid(gate[:, :H].to(F64))[:, :, None]
        got = Q().gemm_head_gate(a.to(DEV), b.to(DEV).contiguous(), gate.to(DEV)[:, :H], H, V, R)
        assert row_err(got, ref.reshape(M, -1)) < tol
    D, T = 8, 6
    q, k, ks, v = rnd(M, H * (D + T), seed=4), rnd(M, H * D, seed=5), rnd(M, T, seed=6), rnd(M, H * V, seed=7)
    sink, mask, out = rnd(H, seed=8), O.visible(M, 0), []
    for a in range(H):
        qa, ka = q[:, a * (D + T):(a + 1) * (D + T)].to(F64), torch.cat([k[:, a * D:(a + 1) * D], ks], 1).to(F64)
        out.append(O.sink_softmax(qa @ ka.T * 0.3, mask, sink[a].to(F64)) @ v[:, a * V:(a + 1) * V].to(F64) * torch.sigmoid(gate[:, a:a + 1].to(F64)))
    got = Q().window_attention_shared(q.to(DEV), k.to(DEV), ks.to(DEV), v.to(DEV), Q().RaggedBatch([(0, M, 0, 0)], DEV), H, 0.3, sink=sink.to(DEV),
                                      gate=gate.to(DEV), gate_per_head=True)
    assert row_err(got, torch.cat(out, 1)) < 2e-5


# ---------------------------------------------------------------------------------------------- products
@pytest.mark.parametrize("M,N,K", [(1, 24, 64), (9, 70, 96), (40, 65, 64), (150, 128, 160), (7, 33, 35), (70, 50, 35)])
def test_activations_of_a_product(M, N, K):
    a, w = rnd(M, K, seed=1), rnd(N, K, seed=2, scale=K ** -0.5)
    cols = N // 3
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 1e-5)):
        z = a.to(dt).to(F64) @ w.to(dt).to(F64).T
        part = torch.cat([O.silu(z[:, :cols]), z[:, cols:]], 1)
        for ref, unary, kw in ((O.relu_squared(z), S().UMBS_UNARY_RELU2, {}), (part, S().UMBS_UNARY_SILU, dict(cols=cols)), (O.silu(z), S().UMBS_UNARY_SILU, {}),
                               (z * -0.35, S().UMBS_UNARY_SCALE, dict(p0=-0.35)), (z, 0, {})):
            assert row_err(Q().gemm_unary(a.to(DEV, dt), w.to(DEV, dt), unary, out_f32=True, **kw), ref) < tol, unary


# ---------------------------------------------------------------------------------------------- routing by token id
@pytest.mark.parametrize("n", [1, 2, 31, 300, 4097])
def test_routing_by_token_id(n):
    vocab = 211
    g = torch.Generator().manual_seed(n)
    shapes = [(1, 1), (5, 3), (8, 2), (300, 7), (6, 6), (1500, 2)] * 6          # more layers than one launch takes
    tables = [torch.rand(vocab, E, generator=g).argsort(-1)[:, :top].to(torch.int32) for E, top in shapes]
    ids = torch.randint(0, vocab, (n,), generator=g).to(torch.int32)
    outs = Q().table_route(ids.to(DEV), [(t.to(DEV).contiguous(), E) for t, (E, _) in zip(tables, shapes)])
    for t, (E, top), (w, off, tok, pos) in zip(tables, shapes, outs):
        chosen = t[ids.long()]                                                    # [n, top]
        w, off, tok, pos = w.cpu(), off.cpu().long(), tok.cpu().long(), pos.cpu().long()
        assert torch.equal(w, torch.full((n, top), 1.0 / top))
        assert torch.equal(off, torch.cat([torch.zeros(1, dtype=torch.long), torch.bincount(chosen.reshape(-1).long(), minlength=E).cumsum(0)]))
        assert torch.equal(pos.sort().values, torch.arange(n * top))              # every pair has a place of its own ...
        assert torch.equal(tok[pos], torch.arange(n * top) // top)                # ... that names its token ...
        e = chosen.reshape(-1).long()
        assert bool(((pos >= off[e]) & (pos < off[e + 1])).all())                 # ... among its expert's pairs


# ---------------------------------------------------------------------------------------------- rows of the stream
@pytest.mark.parametrize("n,width", [(1, 64), (7, 72), (3, 75), (200, 320), (160, 1024), (5, 5000)])
def test_norm_behind_a_block_with_a_multiplier(n, width):
    x, d, w = rnd(n, width, seed=1), rnd(n, width, seed=2, scale=4.0), 1 + 0.2 * rnd(width, seed=3)
    for top in (0, 1, 2, 5, 20):
        kw, total = {}, d.to(F64)
        if top:
            pairs, sel = rnd(n * top, width, seed=4), torch.rand(n, top, generator=torch.Generator().manual_seed(5))
            pos = torch.randperm(n * top, generator=torch.Generator().manual_seed(6)).to(torch.int32)
            total = (sel.to(F64)[:, :, None] * pairs.to(F64)[pos.long()].reshape(n, top, width)).sum(1)
            kw = dict(pair_out=pairs.to(DEV), sel_w=sel.to(DEV), pair_pos=pos.to(DEV))
        ref = x.to(F64) + 0.6 * O.rms_norm(total, w.to(F64), 1e-5)
        for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
            xs, out = x.to(DEV).clone(), torch.empty(n, width, device=DEV, dtype=dt)
            Q().add_rows(xs, out, None if top else d.to(DEV), w.to(DEV), 1e-5, mult=0.6, **kw)
            assert row_err(xs, ref) < 2e-6 and row_err(out, ref) < tol, (top, dt)


def test_embedding_leaves_both_rows():
    table = rnd(50, 72, seed=1)
    ids = torch.tensor([3, 49, 0, 3], dtype=torch.int32)
    for dt in (torch.float32, torch.bfloat16):
        t = table.to(dt)
        y, y2 = Q().embedding_rows(ids.to(DEV), t.to(DEV), 3.5)
        ref = t[ids.long()].float() * 3.5
        assert torch.equal(y.cpu(), ref) and torch.equal(y2.cpu(), ref.to(dt))
