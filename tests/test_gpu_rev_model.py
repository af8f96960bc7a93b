"""The Revudra family on the GPU against the plain oracle (oracle/revudra.py): whole prompts and every layer's stream, the first
tokens, decoding token by token through caches and states, prompts cut into portions, ragged batches, reused slots, long decoding
with a growing cache, window edges decided by one token, other sizes, both dtypes, greedy generation through the engine and its
queue."""
import copy

import pytest
import torch

import rev_helpers as H
from oracle import revudra as O

pytestmark = pytest.mark.gpu


def toks(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.fixture(scope="module")
def mixed():
    t = H.random_tensors(H.MIXED, seed=1)
    return H.MIXED, H.oracle_model(H.MIXED, t), H.product_model(H.MIXED, t, torch.float32)


def run(model, pieces):
    """Feed one sequence as the given portions through a fresh slot; -> logits of every position."""
    slot = model.cache.alloc_slot()
    out = [model.forward([(slot, p, range(len(p)))]) for p in pieces]
    model.cache.free_slot(slot)
    return torch.cat(out)


def cut(seq, sizes):
    out, i = [], 0
    for s in sizes:
        out.append(seq[i:i + s])
        i += s
    if i < len(seq):
        out.append(seq[i:])
    return [p for p in out if p]


def test_whole_prompt_and_layer_streams(mixed):
    cfg, om, pm = mixed
    seq = toks(70, cfg["vocab"], 2)
    ref, streams = O.forward(om, seq)
    slot = pm.cache.alloc_slot()
    got, ly = pm.forward([(slot, seq, range(len(seq)))], layer_out=True)
    pm.cache.free_slot(slot)
    assert ly.shape == streams.shape
    for i in range(len(streams)):
        assert H.close(ly[i], streams[i]), f"layer {i}"
    assert H.close(got, ref)


def test_first_tokens(mixed):
    cfg, om, pm = mixed
    for n in (1, 2, 3, 4):
        seq = toks(n, cfg["vocab"], 10 + n)
        assert H.close(run(pm, [seq]), O.forward(om, seq)[0])
        assert H.close(run(pm, [[x] for x in seq]), O.forward(om, seq)[0])


def test_prefill_then_token_by_token(mixed):
    cfg, om, pm = mixed
    seq = toks(75, cfg["vocab"], 3)
    ref = O.forward(om, seq)[0]
    for first in (1, 2, 9, 17, 30):
        assert H.close(run(pm, [seq[:first]] + [[t] for t in seq[first:]]), ref), first


def test_portions_down_to_two_tokens(mixed):
    cfg, om, pm = mixed
    seq = toks(90, cfg["vocab"], 4)
    ref = O.forward(om, seq)[0]
    # portions shorter and longer than the windows, on and around the tokens the recurrence stages at a time
    for sizes in ([2, 2, 2, 3, 1, 2, 17, 4, 31], [64, 2], [2] * 45, [9, 8, 10, 17, 18], [1, 2, 70], [16, 16, 16, 24], [15, 2, 15, 33, 1], [1, 1, 1, 2, 48]):
        assert H.close(run(pm, cut(seq, sizes)), ref), sizes


def test_unequal_batch_equals_each_alone(mixed):
    cfg, om, pm = mixed
    seqs = [toks(n, cfg["vocab"], 20 + n) for n in (1, 37, 66, 9)]
    tails = [toks(12, cfg["vocab"], 50 + len(s)) for s in seqs]
    refs = [O.forward(om, s + tl)[0] for s, tl in zip(seqs, tails)]
    slots = [pm.cache.alloc_slot() for _ in seqs]
    got = pm.forward([(slots[i], s, range(len(s))) for i, s in enumerate(seqs)])
    o = 0
    for s, r in zip(seqs, refs):
        assert H.close(got[o:o + len(s)], r[:len(s)])
        o += len(s)
    live = list(range(len(seqs)))
    for step in range(12):                             # decode together; one request leaves every fourth step
        if step in (4, 8):
            pm.cache.free_slot(slots[live.pop(1)])
        got = pm.forward([(slots[i], [tails[i][step]], [0]) for i in live])
        for k, i in enumerate(live):
            assert H.close(got[k:k + 1], refs[i][len(seqs[i]) + step][None]), (step, i)
    for i in live:
        pm.cache.free_slot(slots[i])


def test_mixed_step_of_portions_and_single_tokens(mixed):
    """One step may hold a fresh prompt, a later portion and a decoded token side by side."""
    cfg, om, pm = mixed
    a, b, c = toks(40, cfg["vocab"], 31), toks(50, cfg["vocab"], 32), toks(21, cfg["vocab"], 33)
    sa, sb, sc = (pm.cache.alloc_slot() for _ in range(3))
    pm.forward([(sa, a[:39], []), (sb, b[:20], [])])
    got = pm.forward([(sa, a[39:], [0]), (sb, b[20:], range(30)), (sc, c, range(21))])
    assert H.close(got[:1], O.forward(om, a)[0][39:])
    assert H.close(got[1:31], O.forward(om, b)[0][20:])
    assert H.close(got[31:], O.forward(om, c)[0])
    for s in (sa, sb, sc):
        pm.cache.free_slot(s)


def test_freed_slots_are_used_again(mixed):
    """Nothing is cleared on free: the next owner of a slot must not see its predecessor's keys or memories."""
    cfg, om, pm = mixed
    a, b = toks(80, cfg["vocab"], 5), toks(23, cfg["vocab"], 6)
    s = pm.cache.alloc_slot()
    pm.forward([(s, a, [])])
    pm.cache.free_slot(s)
    while pm.cache.alloc_slot() != s:                  # the free list hands slots out in turn
        pass
    ref = O.forward(om, b)[0]
    for first in (1, 7, 23):
        got = torch.cat([pm.forward([(s, b[:first], range(first))])] + [pm.forward([(s, [t], [0])]) for t in b[first:]])
        assert H.close(got, ref)
        pm.cache.free_slot(s)
        while pm.cache.alloc_slot() != s:
            pass
    pm.cache.clear()


def test_long_decoding_with_a_growing_cache():
    """300 tokens, most of them decoded one by one: the latents' caches double under the replayed graph, the windows' rings turn
    over many times, the memories keep their state."""
    cfg = H.MIXED
    t = H.random_tensors(cfg, seed=7)
    om, pm = H.oracle_model(cfg, t), H.product_model(cfg, t, torch.float32, max_tokens=16)
    assert pm.cache.capacity == 16
    seq = toks(300, cfg["vocab"], 8)
    got = run(pm, [seq[:10]] + [[x] for x in seq[10:]])
    assert pm.cache.capacity >= 300
    assert H.close(got, O.forward(om, seq)[0])


def test_a_far_token_stays(mixed):
    """Change one token 200 places back: the oracle's last logits move by far more than the tolerance, and the product's move
    alike, whether those places were a prompt or decoded."""
    cfg, om, pm = mixed
    a = toks(220, cfg["vocab"], 12)
    b = list(a)
    b[3] = (b[3] + 17) % cfg["vocab"]
    ra, rb = O.forward(om, a)[0], O.forward(om, b)[0]
    assert H.row_err(ra[210:], rb[210:]) > 1e-2
    for seq, ref in ((a, ra), (b, rb)):
        assert H.close(run(pm, [seq])[210:], ref[210:])
        assert H.close(run(pm, [seq[:190]] + [[t] for t in seq[190:]])[210:], ref[210:])


@pytest.mark.parametrize("window", [1, 2, 24, 64, 65, 130])
def test_window_edges(window):
    """One attention layer in which token x looks for token y: y at the far end of the window decides x's output, y one place farther
    does not exist -- in prompts, at a portion's start and in decoding."""
    cfg = H.model(48, 97, [H.attention(4, 2, 12, 16, window, 2, base=1e6, scale=4.0, v_mix=True)])
    t = H.random_tensors(cfg, seed=100 + window)
    x, y, n, i = 96, 95, 160, 155
    k = t["l0.mix.k"].roll(24, 1)                      # W_q h = W_k roll(h), and y's embedding is x's rolled: x's query is y's key
    t["l0.mix.q"] = torch.cat([k[:12], k[:12], k[12:], k[12:]])
    t["l0.mix.q.norm"], t["l0.mix.k.norm"] = torch.ones(48), torch.ones(24)
    t["embed"][y] = t["embed"][x].roll(24)
    om, pm = H.oracle_model(cfg, t), H.product_model(cfg, t, torch.float32, graph_decode=False)
    for back in {window - 1, window} - {0}:
        at = i - back
        seq = toks(n, 94, 40)
        seq[i] = x
        other = list(seq)
        seq[at] = y
        diff = H.row_errs(O.forward(om, seq)[0], O.forward(om, other)[0])[i]
        assert (diff > 1e-2) if back < window else (diff < 1e-12)
        ref = O.forward(om, seq)[0]
        for pieces in ([seq], cut(seq, [i]), cut(seq, [at + 1]), [seq[:120]] + [[v] for v in seq[120:]], cut(seq, [150, 2, 3, 2])):
            assert H.close(run(pm, pieces), ref)


def test_values_mix_with_the_first_mixing_layer():
    """The mixed values are what is cached: a later token reads an old token's values in the mix of that token's own source."""
    cfg = H.model(48, 80, [H.attention(2, 1, 8, 12, 30, 4, v_mix=False), H.attention(4, 2, 8, 6, 40, 4), H.lightning(2, 8, 8),
                           H.attention(3, 3, 8, 4, 50, 8), H.attention(6, 1, 8, 12, 60, 2, mlp=H.dense(20))])
    t = H.random_tensors(cfg, seed=4)
    om, pm = H.oracle_model(cfg, t), H.product_model(cfg, t, torch.float32)
    seq = toks(90, cfg["vocab"], 5)
    ref = O.forward(om, seq)[0]
    bare = copy.deepcopy(om)
    for L in bare["layers"]:
        L["mix"]["v_mix"] = False
    assert H.row_err(O.forward(bare, seq)[0], ref) > 1e-2
    assert H.close(run(pm, [seq]), ref)
    assert H.close(run(pm, [seq[:40]] + [[v] for v in seq[40:]]), ref)
    bad = copy.deepcopy(cfg)
    bad["layers"][3]["mixer"]["vdim"] = 6
    with pytest.raises(ValueError):
        H.product_model(bad, H.random_tensors(bad, seed=1), torch.float32)


def test_other_sizes_and_bf16():
    t = H.random_tensors(H.ALIGNED, seed=3)
    om = H.oracle_model(H.ALIGNED, t)
    seq = toks(300, H.ALIGNED["vocab"], 9)
    ref = O.forward(om, seq)[0]
    pm = H.product_model(H.ALIGNED, t, torch.float32)
    assert H.close(run(pm, [seq]), ref)
    assert H.close(run(pm, cut(seq, [140, 2, 1, 1, 30])), ref)
    pb = H.product_model(H.ALIGNED, t, torch.bfloat16)
    whole, parts = run(pb, [seq]), run(pb, [seq[:270]] + [[x] for x in seq[270:]])
    for a, b in ((whole, ref), (parts, ref), (parts, whole)):      # ... and the same numbers however the prompt was cut
        rows = H.row_errs(a, b)
        assert float(rows.median()) < 0.03 and float(rows.max()) < 0.15


def test_bf16_at_sizes_no_tensor_core_tile_takes():
    """bf16 with widths and head sizes that are no multiple of a tile: the products fall back to their plain kernels."""
    cfg, t = H.ODD, H.random_tensors(H.ODD, seed=1)
    om, pb = H.oracle_model(cfg, t), H.product_model(cfg, t, torch.bfloat16)
    seq = toks(120, cfg["vocab"], 41)
    ref = O.forward(om, seq)[0]
    whole, parts = run(pb, [seq]), run(pb, cut(seq, [50, 2, 31])[:3] + [[x] for x in seq[83:]])
    for a, b in ((whole, ref), (parts, ref), (parts, whole)):
        rows = H.row_errs(a, b)
        assert float(rows.median()) < 0.03 and float((rows > 0.15).double().mean()) < 0.05


def test_latents_against_per_head_keys(mixed):
    """A fresh prompt attends over up-projected per-head keys; over the cached latents it gives the same numbers."""
    cfg, om, _ = mixed
    pm = H.product_model(cfg, H.random_tensors(cfg, seed=1), torch.float32, fresh_attention=False)
    seq = toks(66, cfg["vocab"], 43)
    assert H.close(run(pm, [seq]), O.forward(om, seq)[0])


def test_a_table_out_of_range_is_refused():
    cfg = H.model(48, 40, [H.lightning(2, 8, 8, mlp=H.moe(4, 2, 12))])
    t = H.random_tensors(cfg, seed=1)
    for value in (4, -1):
        t["l0.mlp.table"][7, 1] = value
        with pytest.raises(ValueError):
            H.product_model(cfg, t, torch.float32)


def test_greedy_generation_through_engine_and_queue(mixed):
    from umbrella_b200.speculation.auto_engine import AutoEngine
    cfg, om, pm = mixed
    eng = AutoEngine.from_config("cuda:0", engine="batch", model=pm.model_name, dtype="float32", max_batch=2, temperature=0.0)
    eng.initialize()                                   # registry -> config reader -> checkpoint loader
    prompts = [toks(n, cfg["vocab"], 70 + n) for n in (5, 21, 2)]
    outs = eng.generate_batch(prompts, max_new_tokens=6)          # three requests, two slots: two batches
    assert eng.model.cache.live_slots == 0
    assert eng.generate(input_ids=prompts[1], max_new_tokens=6)["generated_tokens"] == outs[1]
    for p, out in zip(prompts, outs):
        seq = list(p)
        for tok in out:
            logits = O.forward(om, seq)[0][-1]
            best = int(logits.argmax())
            if best != tok:                            # only a near tie may differ
                assert float(logits[best] - logits[tok]) < 1e-3
            seq.append(tok)
    eng.update_generation_args(temperature=0.8, topk=8, topp=0.9)
    sampled = eng.generate_batch(prompts[:2], max_new_tokens=5)
    assert all(len(x) == 5 and all(0 <= y < cfg["vocab"] for y in x) for x in sampled)


def _random_config(rng):
    """Sizes, head counts, windows, experts, layer order and constants drawn at random (odd ones included)."""
    layers, vnum = [], rng.choice([12, 24, 60, 128])
    for _ in range(rng.randint(2, 6)):
        kind = rng.choice(["attention", "lightning", "latent"])
        E = rng.choice([1, 2, 5, 9, 40])
        mlp = rng.choice([None, H.dense(rng.choice([16, 30, 128])), H.moe(E, rng.randint(1, min(E, 4)), rng.choice([8, 20, 64]))])
        if kind == "attention":
            kv = rng.choice([g for g in (1, 2, 3, 4) if vnum % g == 0])
            dim = rng.choice([4, 10, 32, 64, 128, 200])
            layers.append(H.attention(kv * rng.choice([1, 2, 5]), kv, dim, vnum // kv, rng.choice([1, 3, 16, 50, 64, 90, 500]),
                                      2 * rng.randint(1, dim // 2), base=rng.choice([50.0, 1e4, 1e6]), v_mix=rng.random() < 0.7, mlp=mlp))
        elif kind == "lightning":
            layers.append(H.lightning(rng.choice([1, 2, 3, 6]), rng.choice([5, 16, 32, 48, 64, 100, 128, 150]), rng.choice([6, 16, 33, 64, 100]), mlp=mlp))
        else:
            layers.append(H.latent(rng.choice([1, 2, 5]), rng.choice([4, 16, 36, 160]), rng.choice([2, 8, 20, 64]), rng.choice([8, 24, 70, 140]),
                                   rng.choice([10, 32, 75]), rng.choice([12, 32, 100, 200]), base=rng.choice([50.0, 1e4, 1e6]), mlp=mlp))
    return H.model(rng.choice([48, 64, 90, 160]), rng.choice([90, 257]), layers, eps=rng.choice([1e-5, 1e-6]), embed=rng.choice([1.0, 5.0, 12.0]),
                   mult=rng.choice([1.0, 0.5, 0.8]), logit=rng.choice([1.0, 0.125, 0.3]))


@pytest.mark.parametrize("seed", [11, 12, 13, 14, 15, 16, 17, 18, 19, 20])
def test_random_configurations(seed):
    """Nothing rests on one model's sizes: random configurations, a ragged batch prefilled and decoded together."""
    import random
    cfg = _random_config(random.Random(seed))
    t = H.random_tensors(cfg, seed=seed)
    om, pm = H.oracle_model(cfg, t), H.product_model(cfg, t, torch.float32, max_tokens=32)
    seqs = [toks(n, cfg["vocab"], seed + n) for n in (120, 41, 87)]
    refs = [O.forward(om, s)[0] for s in seqs]
    slots = [pm.cache.alloc_slot() for _ in seqs]
    cuts = [len(s) - 20 for s in seqs]
    out = pm.forward([(sl, s[:c], range(c)) for sl, s, c in zip(slots, seqs, cuts)])
    got = [[out[sum(cuts[:i]):sum(cuts[:i + 1])]] for i in range(3)]
    for d in range(20):
        o = pm.forward([(sl, [s[c + d]], [0]) for sl, s, c in zip(slots, seqs, cuts)])
        for i in range(3):
            got[i].append(o[i:i + 1])
    for i in range(3):
        assert H.close(torch.cat(got[i]), refs[i]), (seed, i)
