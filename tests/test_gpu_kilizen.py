"""Kilizen on the native sequence engine against the plain oracle (tests/kilizen_oracle.py): every mechanism alone, then whole models
through prompts, decoding, portions, mixed batches, reused slots and pages, the scheduler and the command line.  Configurations and
weights are made here; none of them has the sizes of a published model."""
import json

import numpy as np
import pytest
import torch

import kilizen_oracle as O

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------------------------ configurations
def ffd(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, shared=20):
    f = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def rope(dims, base=1000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def win(heads=4, kv=2, dim=16, scale=0.25, size=9, keep=3, rot=(8, 1000.0, (3.0, 24, 16.0, 2.0)), mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": size, "keep_first": keep}, "rot": rope(*rot)}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def full(heads=4, kv=2, dim=12, vdim=10, scale=0.3, rot=(12, 500.0), mlp=None):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": rope(*rot)}, "mlp": mlp}


def mem(heads=2, dim=8, vdim=12, cap=5.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def config(layers, width=48, vocab=61, eps=2e-5, loop=None):
    cfg = {"architecture": "Kilizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# Layer orders, loops, head groupings, router sizes and constants all differ between them.
CFG_MIXED = config([full(mlp=ffd(40)), win(mlp=moe()), mem(mlp=moe(experts=5, top=3, ff=28, shared=16)), win(heads=2, kv=1, size=5, keep=7, rot=(4, 50.0), mlp=None), mem(heads=3, dim=10, vdim=6, cap=2.0)],
                   loop=(1, 3, 2))
# nothing a multiple of 8, one head, one key/value head for all, a window of one token, a loop of one layer that ends the stack, a router that
# takes every expert, no shared expert
CFG_ODD = config([win(heads=3, kv=1, dim=6, scale=0.5, size=1, keep=1, rot=(2, 20.0), mlp=moe(experts=3, top=3, ff=13, shared=0)), mem(heads=1, dim=5, vdim=7, cap=30.0, mlp=ffd(21)),
                  full(heads=1, kv=1, dim=5, vdim=9, scale=0.6, rot=(4, 30.0), mlp=moe(experts=7, top=1, ff=11, shared=9))],
                 width=36, vocab=33, eps=1e-3, loop=(2, 3, 3))
# sizes that the tensor-core kernels take; the loop covers the whole stack
CFG_WIDE = config([win(heads=8, kv=2, dim=64, scale=0.125, size=37, keep=5, rot=(32, 10000.0, (4.0, 64, 32.0, 1.0)), mlp=moe(experts=10, top=4, ff=64, shared=96)),
                   full(heads=6, kv=3, dim=32, vdim=48, scale=0.2, rot=(32, 10000.0), mlp=ffd(160)), mem(heads=2, dim=32, vdim=64, cap=10.0, mlp=moe(experts=4, top=2, ff=72, shared=40))],
                  width=128, vocab=150, loop=(0, 3, 2))
CONFIGS = {"mixed": CFG_MIXED, "odd": CFG_ODD, "wide": CFG_WIDE}


def make_weights(cfg, seed, **kw):
    """name -> float32 array whose values are exactly representable in bfloat16 (so both engine dtypes hold the same model)."""
    return {k: v.numpy() for k, v in O.random_weights(cfg, seed, **kw).items()}


def build(cfg, weights, dtype="float32", max_tokens=256, slots=4, page_size=4, max_step_tokens=64):
    from wf_bitnet import registry
    model = registry.resolve(cfg)(cfg, dtype=dtype, max_tokens=max_tokens, slots=slots, page_size=page_size, max_step_tokens=max_step_tokens)
    model.load_weights((k, v, "F32") for k, v in weights.items())
    return model


def t64(weights):
    return {k: torch.from_numpy(np.asarray(v)).double() for k, v in weights.items()}


def oracle_logits(cfg, weights, tokens, streams=None):
    return O.forward(cfg, t64(weights), list(tokens), streams).numpy()


def rel_err(got, want):
    """per row: RMS of the difference (mean taken off) over the RMS of the expected row"""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / (np.sqrt((want ** 2).mean(-1)) + 1e-12)


TOL = {"float32": 2e-4, "bfloat16": 6e-2}


def assert_close(got, want, dtype, what, factor=1.0):
    """float32: every row within tolerance.  bfloat16: a position where the random model happens to be ill-conditioned (two keys or two
    experts that nearly tie, a state that is still almost empty) multiplies the rounding of the layers below it; such positions are few, so
    four rows in five must be within tolerance, the typical row well within it, and none far off."""
    err = rel_err(np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64))
    if dtype == "float32" or err.size <= 4:
        assert err.max() < factor * TOL[dtype], (what, int(err.argmax()), float(err.max()))
    else:
        assert (err < factor * TOL[dtype]).mean() >= 0.8 and np.median(err) < 0.5 * TOL[dtype] and err.max() < 0.5, (what, int(err.argmax()), float(err.max()), float(np.median(err)))


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def bf16_exact(a):
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy()


def _rows(n, W, seed, scale=1.0):
    return bf16_exact(np.random.default_rng(seed).standard_normal((n, W)) * scale)


def run_alone(m, tokens, cuts):
    """one request through the engine in portions `cuts`; logits of every position"""
    s = m.admit()
    out, a = [], 0
    for c in cuts:
        out.append(m.step([s], [c], tokens[a:a + c], list(range(c))))
        a += c
    m.release(s)
    return np.concatenate(out)


def part_alone(m, layer, part, rows, cuts):
    """one part of one layer run on given rows, in portions, through the cache and state of one slot"""
    s = m.admit()
    out, a = [], 0
    for c in cuts:
        out.append(m.engine.run_part(layer, part, [s], [c], rows[a:a + c]))
        a += c
    m.release(s)
    return np.concatenate(out)


def oracle_mixer(cfg, w, li, rows):
    L = cfg["layers"][li]
    return O.MIXERS[L["type"]](torch.from_numpy(rows).double(), t64(w), f"l{li}.mix.", L["mixer"], cfg["norm"]["eps"]).numpy()


# ---------------------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixers_alone_whole_and_in_portions(name, dtype):
    """Every layer run's mixer on random rows (a repeated layer once per pass, each with its own cache): as one portion, in portions of
    1 / 2 / 3 / ... tokens through cache and state, and token by token."""
    cfg = CONFIGS[name]
    w = make_weights(cfg, 11)
    m = build(cfg, w, dtype, max_tokens=512)
    n = 45
    runs = O.layer_runs(cfg)
    assert m.engine.layer_runs() == len(runs)
    for ri, (li, _) in enumerate(runs):
        rows = _rows(n, cfg["width"], 20 + ri)
        want = oracle_mixer(cfg, w, li, rows)
        for cuts in ([n], [1, 2, 3, 5, 7, 2, 11, 14], [1] * n):
            assert_close(part_alone(m, ri, 2, rows, cuts), want, dtype, (name, ri, cuts[:3]))
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_four_norms_of_a_layer(dtype):
    """Element-wise norms, with inputs small and large against 1 / alpha and alphas of either sign."""
    for W in (40, 37):
        cfg = config([mem(mlp=ffd(24))], width=W)
        w = make_weights(cfg, 41)
        w["l0.norm1b.alpha"] = bf16_exact(-1.75)
        m = build(cfg, w, dtype)
        tw = t64(w)
        for scale in (0.1, 3.0):
            rows = _rows(9, W, 42, scale)
            h = torch.from_numpy(rows).double()
            for part, nm in ((0, "norm1"), (5, "norm2"), (6, "norm1b"), (7, "norm2b")):
                assert_close(part_alone(m, 0, part, rows, [9]), O.dyn_tanh(h, tw, f"l0.{nm}").numpy(), "float32", (nm, scale))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_feed_forwards_alone(dtype):
    """Dense and routed, with and without a shared expert, sizes aligned and not, at row counts that take every form of the product
    (few-row streams, mma.sync, tcgen05, per-pair experts, grouped experts)."""
    for W, f in ((48, ffd(56)), (40, ffd(33)), (48, moe(experts=9, top=3, ff=32, shared=40)), (64, moe(experts=5, top=5, ff=24, shared=0)), (36, moe(experts=7, top=1, ff=11, shared=9)),
                 (128, moe(experts=40, top=6, ff=64, shared=24))):
        cfg = config([mem(mlp=f)], width=W)
        w = make_weights(cfg, 43)
        m = build(cfg, w, dtype, max_step_tokens=256)
        for n in (1, 3, 7, 12, 30, 150):
            rows = _rows(n, W, 44 + n, 1.5)
            want = O.feed_forward(torch.from_numpy(rows).double(), t64(w), "l0.mlp.", f).numpy()
            assert_close(part_alone(m, 0, 3, rows, [n]), want, dtype, (W, f["kind"], n))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_router_weights_and_choice(dtype):
    """Hand-made logits: the weights are a softmax over the chosen logits (not over all), a large common offset changes nothing, and two
    logits closer than bfloat16 resolves are told apart."""
    W, E = 32, 4
    cfg = config([mem(mlp=moe(experts=E, top=2, ff=8, shared=0))], width=W)
    w = make_weights(cfg, 45)
    w["l0.mlp.router"] = np.zeros((E, W), dtype=np.float32)
    for e in range(E):
        w["l0.mlp.router"][e, e] = 1.0
    f = cfg["layers"][0]["mlp"]
    rows = _rows(3, W, 46)
    rows[0, :E] = [1.0, 0.5, -1.0, 0.25]
    rows[1, :E] = [60.0, 61.0, 59.0, 60.5]
    rows[2, :E] = [-3.0, -2.5, -40.0, -60.0]
    m = build(cfg, w, dtype)
    assert_close(part_alone(m, 0, 3, rows, [3]), O.feed_forward(torch.from_numpy(rows).double(), t64(w), "l0.mlp.", f).numpy(), dtype, "weights")
    close = rows.copy()
    close[:, :E] = [[1.0, -2.0, 0.7501, 0.75], [1.0, -2.0, 0.75, 0.7501], [-9.0, 3.0, 2.0001, 2.0]]        # bfloat16 neighbours of 0.75 are 0.004 apart
    want = O.feed_forward(torch.from_numpy(close).double(), t64(w), "l0.mlp.", f).numpy()
    assert rel_err(want[1:2], want[0:1]).max() > 0.05
    assert_close(part_alone(m, 0, 3, close, [3]), want, dtype, "close call")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_rotation_of_every_extent_and_scaling(dtype):
    """No rotation, two entries, all entries; interpolation with ramps of different width and place, at positions up to 2000."""
    far = [(24, 1e4, (8.0, 256, 32.0, 1.0)), (24, 100.0, (2.0, 4096, 4.0, 3.9)), (2, 30.0), (24, 5e5), (10, 1000.0, (1.0, 64, 8.0, 1.0)), (0, 10.0)]
    for k, rot in enumerate(far):
        for layer in (win(heads=2, kv=1, dim=24, size=30, keep=2, rot=rot), full(heads=2, kv=2, dim=24, vdim=16, rot=rot)):
            cfg = config([layer], width=32)
            w = make_weights(cfg, 47 + k)
            n = 2000 if k == 0 else 90
            rows = _rows(n, 32, 48)
            want = oracle_mixer(cfg, w, 0, rows)
            m = build(cfg, w, dtype, max_tokens=2048, page_size=16, max_step_tokens=2048)
            assert_close(part_alone(m, 0, 2, rows, [n - 3, 1, 2]), want, dtype, (rot, layer["type"]))
            m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_take_weight(dtype):
    """Learned sinks, large for some heads: leaving them out would move the output by tens of percent."""
    for layer in (win(heads=4, kv=2, dim=8, scale=0.1, size=5, keep=2, rot=(4, 50.0)), full(heads=4, kv=1, dim=8, vdim=6, scale=0.1, rot=(8, 50.0))):
        cfg = config([layer], width=32)
        w = make_weights(cfg, 171)
        w["l0.mix.sink"] = bf16_exact(np.array([3.0, -1.0, 1.5, 40.0]))
        rows = _rows(24, 32, 172)
        want = oracle_mixer(cfg, w, 0, rows)
        none = dict(w)
        none["l0.mix.sink"] = np.full(4, -60.0, dtype=np.float32)
        if layer["type"] == "attention":
            assert rel_err(oracle_mixer(cfg, none, 0, rows), want).min() > 0.1
        m = build(cfg, w, dtype)
        for cuts in ([24], [1] * 24, [5, 2, 17]):
            assert_close(part_alone(m, 0, 2, rows, cuts), want, dtype, (layer["type"], cuts[:2]))
        m.close()


# ------------------------------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_decode_and_portions_agree_with_the_oracle(name, dtype):
    cfg = CONFIGS[name]
    w = make_weights(cfg, 51)
    m = build(cfg, w, dtype, max_tokens=512)
    n = 61
    toks = tokens_for(cfg, n, 52)
    want = oracle_logits(cfg, w, toks)
    for cuts in ([n], [1] * n, [40] + [1] * 21, [2, 2, 3, 2, 5, 7, 11, 2, 13, 14], [17, 1, 1, 19, 1, 22]):
        assert_close(run_alone(m, toks, cuts), want, dtype, (name, cuts[:4]), 1.5)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_streams_and_first_positions(dtype):
    """Prompts of one to five tokens: the stream after every layer run (before the embedding of a repeated pass is added) and the logits."""
    for name in ("odd", "mixed", "wide"):
        cfg = CONFIGS[name]
        w = make_weights(cfg, 61)
        m = build(cfg, w, dtype)
        for n in (1, 2, 3, 4, 5):
            toks = tokens_for(cfg, n, 62 + n)
            streams = []
            want = oracle_logits(cfg, w, toks, streams)
            s = m.admit()
            out, tap = m.engine.step_with_layer_tap([s], [n], toks, list(range(n)))
            m.release(s)
            assert len(tap) == len(streams)
            for ri, st in enumerate(streams):
                assert_close(tap[ri], st.numpy(), dtype, ("stream", n, ri))
            assert_close(out, want, dtype, ("logits", n))
            assert_close(run_alone(m, toks, [n]), want, dtype, ("logits without taps", n))
        m.close()


def test_loops_of_every_shape():
    """Loops at the start, in the middle, at the end and over the whole stack, one to four passes; taking the embedding out of the second
    pass, or a pass reading another's cache, would show (the oracle without a loop, or with the layers merely repeated, is far off)."""
    layers = [win(size=6, keep=2), mem(mlp=ffd(24)), full(mlp=moe())]
    toks = None
    for loop in (None, (0, 1, 2), (1, 2, 3), (1, 3, 2), (0, 3, 4), (2, 3, 2), (0, 2, 1)):
        cfg = config(layers, loop=loop)
        w = make_weights(cfg, 65)
        toks = toks or tokens_for(cfg, 33, 66)
        want = oracle_logits(cfg, w, toks)
        if loop and loop[2] > 1:
            once = oracle_logits(config(layers), w, toks)
            x = t64(w)["embed"][torch.tensor(toks)]
            for i, _ in O.layer_runs(cfg):
                x = O.layer(x, t64(w), i, layers[i], cfg["norm"]["eps"])
            plain = (O.dyn_tanh(x, t64(w), "final.norm") @ t64(w)["head"].T).numpy()
            assert np.median(rel_err(once, want)) > 0.05 and np.median(rel_err(plain, want)) > 0.05
        m = build(cfg, w, "float32")
        for cuts in ([33], [20] + [1] * 13, [2, 9, 1, 21]):
            assert_close(run_alone(m, toks, cuts), want, "float32", (loop, cuts[:3]))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_each_request_alone(dtype):
    """Four unequal requests advance together — portions of some beside single tokens of others, one of them paused for a step — and
    every position equals the oracle of its request alone."""
    for name in ("mixed", "wide"):
        cfg = CONFIGS[name]
        w = make_weights(cfg, 71)
        m = build(cfg, w, dtype, max_tokens=512)
        reqs = [tokens_for(cfg, n, 72 + n) for n in (37, 9, 23, 50)]
        want = [oracle_logits(cfg, w, r) for r in reqs]
        plan = [[5, 9, 1, 20], [1, 0, 2, 1], [13, 0, 1, 1], [1, 0, 0, 7], [17, 0, 19, 21]]
        slots = [m.admit() for _ in reqs]
        fed = [0] * 4
        for step in plan:
            sl, cn, tk, rows = [], [], [], []
            for i, c in enumerate(step):
                if c:
                    sl.append(slots[i]); cn.append(c); tk += reqs[i][fed[i]:fed[i] + c]
                    rows += [(i, fed[i] + k) for k in range(c)]
                    fed[i] += c
            out = m.step(sl, cn, tk, list(range(len(tk))))
            assert_close(out, np.stack([want[i][p] for i, p in rows]), dtype, (name, step), 1.5)
        assert fed == [len(r) for r in reqs]
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_are_used_again(dtype):
    """Six requests through a pool of 12 pages and 2 slots, a neighbour stepping in between: a slot's recurrent states (one per pass of the
    loop) and a page's rows must not leak into the next request."""
    cfg = CONFIGS["mixed"]
    w = make_weights(cfg, 81)
    m = build(cfg, w, dtype, max_tokens=48, slots=2, page_size=4)
    other = m.admit()
    filler = tokens_for(cfg, 40, 82)
    used = 0
    for k, n in enumerate((19, 7, 24, 1, 13, 22)):
        toks = tokens_for(cfg, n, 83 + k)
        want = oracle_logits(cfg, w, toks)
        s = m.admit()
        assert s >= 0
        half = n // 2
        got = []
        if half:
            got.append(m.step([s], [half], toks[:half], list(range(half))))
        if used + 2 > 20:                          # the neighbour starts over before it outgrows its share of the pool
            m.release(other); other = m.admit(); used = 0
        m.step([other], [2], filler[used:used + 2], [])
        used += 2
        got.append(m.step([s], [n - half], toks[half:], list(range(n - half))))
        assert_close(np.concatenate(got), want, dtype, (k, n), 1.5)
        m.release(s)
    assert m.free_slots() == 1
    m.close()


# --------------------------------------------------------------------------------------------- one key that decides, at every edge
def _half_matrix(rows, W, seed):
    return _rows(rows, W // 2, seed, 1.0 / np.sqrt(W // 2))


def _deciding_model(dtype, layer, page_size, n):
    """One attention layer whose keys read the first half of the input row and whose queries read the second half through the SAME matrix:
    a probe row that carries in its second half what a marked row carries in its first meets that key with the largest score there is
    (sharp softmax, few rotated entries); its own key is an ordinary one."""
    W, mx = 64, layer["mixer"]
    cfg = config([layer], width=W)
    w = make_weights(cfg, 91)
    A = _half_matrix(mx["dim"], W, 92)
    w["l0.mix.k"] = np.concatenate([A, np.zeros_like(A)], 1)
    w["l0.mix.q"] = np.concatenate([np.concatenate([np.zeros_like(A), A], 1)] * mx["heads"], 0)
    for b in ("q.b", "k.b"):
        if "l0.mix." + b in w:
            w["l0.mix." + b] = np.zeros_like(w["l0.mix." + b])
    return cfg, w, build(cfg, w, dtype, max_tokens=n + 64, page_size=page_size, max_step_tokens=n + 8)


def _marked_rows(n, probe, marked, seed):
    rows = _rows(n, 64, seed)
    rows[probe, 32:] = rows[marked, :32]
    return rows


def _cuts(points, n):
    edges = sorted({p for p in points if 0 < p < n} | {0, n})
    return [b - a for a, b in zip(edges, edges[1:])]


def _check_marked(cfg, w, m, dtype, n, probe, marked, what):
    rows = _marked_rows(n, probe, marked, 93)
    want = oracle_mixer(cfg, w, 0, rows)
    for points in ((), (probe, probe + 1), (marked, marked + 2, probe), (marked + 1, probe)):
        cuts = _cuts(points, n)
        got = part_alone(m, 0, 2, rows, cuts)
        assert_close(got[probe:probe + 1], want[probe:probe + 1], dtype, (what, cuts), 2.0)
        if dtype == "float32":                 # in bfloat16 two ordinary keys that nearly tie under the sharp softmax may swap
            assert_close(got, want, dtype, (what, cuts, "all"), 2.0)
    return want[probe]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,keep,page_size,n,probe_back", [(6, 3, 4, 40, 0), (37, 5, 4, 90, 1), (300, 20, 16, 400, 2), (64, 64, 16, 200, 3), (16, 70, 16, 170, 0), (600, 130, 64, 900, 0),
                                                              (33, 1, 16, 100, 0)])
def test_a_deciding_key_at_every_edge_of_window_and_kept_positions(dtype, size, keep, page_size, n, probe_back):
    """The marked key sits on the last position the window still reaches or one before it, on the last kept first position or the next one,
    on position 0, and near; the probe comes at the end of a prompt, in the middle of a portion, as a single decoded token, and after
    portions cut at the marked key.  Neighbouring placements differ by tens of percent in the oracle, so an edge one token off cannot pass."""
    cfg, w, m = _deciding_model(dtype, win(heads=2, kv=1, dim=64, scale=0.5, size=size, keep=keep, rot=(4, 1e4, (2.0, 64, 8.0, 1.0))), page_size, n)
    probe = n - 1 - probe_back
    first_seen = probe - size + 1
    assert first_seen - 1 > keep
    outs = {k: _check_marked(cfg, w, m, dtype, n, probe, at, (size, keep, k))
            for k, at in (("window in", first_seen), ("window out", first_seen - 1), ("kept in", keep - 1), ("kept out", keep), ("start", 0), ("near", probe - 1))}
    for a, b in (("window in", "window out"), ("kept in", "kept out")):
        gap = np.linalg.norm(outs[a] - outs[b]) / np.linalg.norm(outs[a])
        assert gap > 0.3, (a, gap)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size,n,marked", [(64, 400, 0), (64, 400, 1), (64, 400, 63), (64, 400, 64), (64, 400, 65), (16, 330, 127), (16, 330, 128), (4, 90, 3)])
def test_a_far_key_decides_in_causal_attention(dtype, page_size, n, marked):
    """One key hundreds of positions back, on both sides of page borders and on the very first positions, is the one the last query
    wants; a reader blind to that position differs by tens of percent."""
    cfg, w, m = _deciding_model(dtype, full(heads=2, kv=1, dim=48, vdim=40, scale=0.6, rot=(4, 1e5)), page_size, n)
    probe = n - 1
    rows = _marked_rows(n, probe, marked, 93)
    blind = rows.copy()
    blind[marked] = _rows(1, 64, 99)[0]
    assert rel_err(oracle_mixer(cfg, w, 0, blind)[probe:], oracle_mixer(cfg, w, 0, rows)[probe:]).max() > 0.3
    _check_marked(cfg, w, m, dtype, n, probe, marked, marked)
    m.close()


def test_state_is_carried_over_hundreds_of_tokens():
    """A forget gate of almost one: 300 tokens in seven portions with a neighbour stepping in another slot.  A state that lost its first
    half would move the last outputs by more than a tenth."""
    cfg = config([mem(heads=2, dim=16, vdim=8, cap=8.0)], width=32)
    w = make_weights(cfg, 101)
    w["l0.mix.f.b"] = np.full_like(w["l0.mix.f.b"], 6.0)
    n = 300
    rows = _rows(n, 32, 102)
    want = oracle_mixer(cfg, w, 0, rows)
    assert rel_err(oracle_mixer(cfg, w, 0, rows[150:])[-20:], want[-20:]).max() > 0.1
    for dtype in ("float32", "bfloat16"):
        m = build(cfg, w, dtype, max_tokens=1024, max_step_tokens=128)
        s, nb = m.admit(), m.admit()
        out, a = [], 0
        for c in (3, 64, 1, 100, 2, 90, 40):
            out.append(m.engine.run_part(0, 2, [s], [c], rows[a:a + c]))
            m.engine.run_part(0, 2, [nb], [5], _rows(5, 32, 103 + a))
            a += c
        assert_close(np.concatenate(out), want, dtype, dtype, 2.0)
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_in_a_ragged_batch(dtype):
    """A long, a short and a chunk-sized portion in three slots, after portions of other sizes: the recurrence runs in parallel pieces, the
    attention's prompt tiles span windows and the gap behind the kept first positions."""
    for layer in (mem(heads=3, dim=12, vdim=10, cap=6.0), win(heads=4, kv=2, dim=32, size=70, keep=9, rot=(8, 1e4)), full(heads=4, kv=4, dim=24, vdim=32, rot=(24, 1e4))):
        cfg = config([layer], width=32)
        w = make_weights(cfg, 161)
        m = build(cfg, w, dtype, max_tokens=4096, page_size=16, max_step_tokens=1024)
        rows = [_rows(n, 32, 162 + n) for n in (37 + 600, 5 + 128, 300 + 1)]
        want = [oracle_mixer(cfg, w, 0, r) for r in rows]
        assert_close(part_alone(m, 0, 2, rows[0], [37, 600]), want[0], dtype, "one slot", 2.0)
        slots = [m.admit() for _ in rows]
        got = m.engine.run_part(0, 2, slots, [37, 5, 300], np.concatenate([rows[0][:37], rows[1][:5], rows[2][:300]]))
        got2 = m.engine.run_part(0, 2, slots, [600, 128, 1], np.concatenate([rows[0][37:], rows[1][5:], rows[2][300:]]))
        assert_close(np.concatenate([got, got2]), np.concatenate([want[0][:37], want[1][:5], want[2][:300], want[0][37:], want[1][5:], want[2][300:]]), dtype, "ragged", 2.0)
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_over_page_borders(dtype):
    """150 decoded tokens on 4-token pages: windows slide over decoded tokens only, rotation angles grow, every pass of the loop decodes
    through its own cache."""
    cfg = CONFIGS["mixed"]
    w = make_weights(cfg, 121)
    m = build(cfg, w, dtype, max_tokens=256, page_size=4)
    toks = tokens_for(cfg, 160, 122)
    assert_close(run_alone(m, toks, [10] + [1] * 150), oracle_logits(cfg, w, toks), dtype, "decode", 1.5)
    m.close()


def test_tensor_core_attention_with_key_splits_in_a_ragged_batch():
    """bfloat16, sizes the tensor-core kernels take, contexts long enough that decoding cuts the keys (kept first ones, then the window)
    over several blocks: three sequences of unequal length, prompts in portions and then decoded together; float32 (the plain kernels)
    beside it."""
    cfg = config([win(heads=8, kv=2, dim=64, scale=0.125, size=520, keep=77, rot=(16, 1e4)), full(heads=8, kv=1, dim=96, vdim=64, scale=0.1, rot=(96, 1e4))], width=64, vocab=90)
    w = make_weights(cfg, 131)
    lens = (770, 300, 41)
    reqs = [tokens_for(cfg, n + 6, 132 + n) for n in lens]
    want = [oracle_logits(cfg, w, r) for r in reqs]
    for dtype in ("bfloat16", "float32"):
        m = build(cfg, w, dtype, max_tokens=1300, page_size=16, max_step_tokens=640)
        slots = [m.admit() for _ in reqs]
        for i, n in enumerate(lens):
            a = 0
            for c in (n // 3, n - n // 3):
                out = m.step([slots[i]], [c], reqs[i][a:a + c], list(range(c)))
                assert_close(out, want[i][a:a + c], dtype, ("prompt", i, a), 1.5)
                a += c
        for k in range(6):
            out = m.step(slots, [1, 1, 1], [reqs[i][lens[i] + k] for i in range(3)], [0, 1, 2])
            assert_close(out, np.stack([want[i][lens[i] + k] for i in range(3)]), dtype, ("decode", k), 1.5)
        m.close()


def _random_config(rng):
    """1-4 layers of random kinds with sizes drawn independently of each other, often with a loop"""
    W = rng.choice([24, 40, 72, 96, 136, 200])

    def mlp():
        k = rng.choice(["none", "dense", "moe", "moe"])
        if k == "none":
            return None
        if k == "dense":
            return ffd(rng.choice([W, rng.randint(8, 3 * W)]))
        E = rng.choice([1, 3, 8, 20])
        return moe(experts=E, top=rng.randint(1, min(E, 6)), ff=rng.choice([16, 40, rng.randint(5, 90)]), shared=rng.choice([0, 24, rng.randint(5, 90)]))

    def scaling():
        return rng.choice([None, (rng.choice([1.5, 2.0, 8.0]), rng.choice([16, 200, 4096]), rng.choice([32.0, 8.0]), rng.choice([1.0, 0.5]))])

    layers = []
    n = rng.randint(1, 4)
    for _ in range(n):
        kind = rng.choice(["attention", "attention_2", "mlstm"])
        G, rep, d = rng.choice([1, 2, 3]), rng.choice([1, 2, 4, 7, 8]), rng.choice([6, 16, 24, 64, 96, 128, 192])
        rot = (2 * rng.randint(1, d // 2), rng.choice([100.0, 10000.0, 5e5]), scaling())
        if kind == "attention":
            layers.append(win(heads=G * rep, kv=G, dim=d, scale=rng.choice([d ** -0.5, 0.2]), size=rng.choice([1, 2, 7, 16, 50, 120]), keep=rng.choice([0, 1, 4, 64, 65, 150]), rot=rot, mlp=mlp()))
        elif kind == "attention_2":
            layers.append(full(heads=G * rep, kv=G, dim=d, vdim=rng.choice([8, 20, 48, 128, 136]), scale=rng.choice([d ** -0.5, 0.1]), rot=rot, mlp=mlp()))
        else:
            layers.append(mem(heads=rng.choice([1, 2, 5]), dim=rng.choice([4, 16, 33, 72, 160]), vdim=rng.choice([4, 24, 40, 136]), cap=rng.choice([1.5, 9.0, 25.0]), mlp=mlp()))
    a = rng.randint(0, n - 1)
    loop = rng.choice([None, (a, rng.randint(a + 1, n), rng.choice([1, 2, 3]))])
    return config(layers, width=W, vocab=rng.choice([50, 97, 300]), eps=rng.choice([1e-6, 1e-4]), loop=loop)


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations(seed):
    """Layer orders, loops, head counts, sizes, windows and constants drawn at random: one prompt whole, prompt + decoded tail, and in
    random portions, in both dtypes."""
    import random
    rng = random.Random(3000 + seed)
    cfg = _random_config(rng)
    n = rng.choice([3, 17, 64, 130, 290])
    w = make_weights(cfg, 200 + seed)
    toks = tokens_for(cfg, n, 300 + seed)
    want = oracle_logits(cfg, w, toks)
    k = max(1, n - rng.randint(1, 8))
    cuts, left = [], n
    while left:
        cuts.append(min(left, rng.choice([1, 2, 3, 5, 16, 33, 64, 100])))
        left -= cuts[-1]
    for dtype in ("float32", "bfloat16"):
        m = build(cfg, w, dtype, max_tokens=512, page_size=rng.choice([4, 16, 64]), max_step_tokens=512)
        for c in ([n], [k] + [1] * (n - k), cuts):
            assert_close(run_alone(m, toks, c), want, dtype, (seed, dtype, c[:4]), 1.5)
        m.close()


# ------------------------------------------------------------------------------------------------- scheduler and command line
def _greedy_matches(cfg, w, prompt, output):
    seq = list(prompt)
    for t in output:
        lg = oracle_logits(cfg, w, seq)[-1]
        top2 = np.sort(lg)[-2:]
        if top2[1] - top2[0] > 1e-3 * np.abs(lg).max():
            assert int(np.argmax(lg)) == t
        seq.append(t)


def test_greedy_generation_through_the_scheduler():
    from wf_bitnet.scheduler import Request, Scheduler
    cfg = CONFIGS["mixed"]
    w = make_weights(cfg, 141)
    m = build(cfg, w, "float32", max_tokens=96, slots=2, page_size=4, max_step_tokens=16)
    sched = Scheduler(m, max_prefill_chunk=5)
    prompts = [tokens_for(cfg, n, 142 + n) for n in (11, 3, 17, 6, 1)]
    for i, p in enumerate(prompts):
        sched.add(Request(f"r{i}", p, max_new_tokens=6))
    done = {r.rid: r for r in sched.run()}
    assert len(done) == 5 and m.free_slots() == 2
    for i, p in enumerate(prompts):
        _greedy_matches(cfg, w, p, done[f"r{i}"].output)
    m.close()


def _write_model_dir(path, cfg, weights):
    import struct
    header, blob = {}, b""
    for name, a in weights.items():
        a = np.asarray(a, dtype=np.float32)
        raw = torch.from_numpy(a.copy()).to(torch.bfloat16).view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    h = json.dumps(header).encode()
    (path / "config.json").write_text(json.dumps(cfg))
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + blob)


def test_command_line_trace_replay_and_generate(tmp_path):
    """`trace` (bin/trace_run) replays a schedule with mixed batches, a pause, and a finished request whose slot and pages go to the next
    one; `generate` runs the scheduler.  The model class comes from config.json."""
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    cfg = CONFIGS["mixed"]
    w = make_weights(cfg, 151)
    _write_model_dir(tmp_path, cfg, w)
    reqs = {"a": tokens_for(cfg, 21, 152), "b": tokens_for(cfg, 9, 153), "c": tokens_for(cfg, 14, 154)}
    want = {k: oracle_logits(cfg, w, v) for k, v in reqs.items()}
    plan = [[("a", 6)], [("a", 1), ("b", 8)], [("a", 10), ("b", 1)], [("a", 4)], [("c", 2)], [("c", 11)], [("c", 1)]]
    fed, lines, expect = {k: 0 for k in reqs}, [], []
    for n, step in enumerate(plan):
        ents, end, rows = [], [], []
        for rid, c in step:
            ents.append({"id": rid, "tokens": reqs[rid][fed[rid]:fed[rid] + c], "want": list(range(c))})
            rows += [(rid, fed[rid] + k) for k in range(c)]
            fed[rid] += c
            if fed[rid] == len(reqs[rid]):
                end.append(rid)
        lines.append(json.dumps({"step": n, "entries": ents, "end": end}))
        expect.append(rows)
    out = tmp_path / "out"
    out.mkdir()
    for dtype in ("float32", "bfloat16"):
        r = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "64", "--slots", "2"],
                           input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done ")] == [f"done {n}" for n in range(len(plan))]
        got = [np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]) for n, rows in enumerate(expect)]
        assert_close(np.concatenate(got), np.stack([want[rid][pos] for rows in expect for rid, pos in rows]), dtype, dtype, 1.5)
    r = subprocess.run([sys.executable, "-m", "wf_bitnet.cli", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "5",
                        "--prompt-ids", ",".join(map(str, reqs["a"])), "--prompt-ids", ",".join(map(str, reqs["b"])), "--slots", "1", "--prefill-chunk", "4"],
                       capture_output=True, text=True, timeout=600, env=dict(__import__("os").environ, PYTHONPATH=str(root / "wrinklefree-inference-engine_b200")))
    assert r.returncode == 0, r.stderr[-2000:]
    outs = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    assert [o["id"] for o in outs] == ["r0", "r1"]
    for o, rid in zip(outs, ("a", "b")):
        _greedy_matches(cfg, w, reqs[rid], o["output_ids"])
