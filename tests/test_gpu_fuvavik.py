"""Fuvavik on the native sequence engine against the plain oracle (tests/fuvavik_oracle.py): every mechanism alone, then whole models
through prompts, decoding, portions, mixed batches, reused slots and pages, the scheduler and the command line.  Configurations and
weights are made here; none of them has the sizes of a published model."""
import json

import numpy as np
import pytest
import torch

import fuvavik_oracle as O

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------------------------ configurations
def par(heads=4, kv=2, dim=16, vdim=24, scale=0.3, window=9, rh=3, rd=8, rv=12, tau=8.0, ff=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        left["mask"] = {"size": window}
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": rh, "dim": rd, "vdim": rv, "tau": tau}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=48, vocab=61, eps=2e-5, escale=1.7, positions=420, cap=12.0):
    return {"architecture": "Fuvavik", "vocab": vocab, "width": width, "embedding": {"scale": escale}, "norm": {"eps": eps}, "max_positions": positions,
            "logit_softcap": cap, "layers": layers}


# (config, inner sizes of the decay projections).  Head groupings, sizes, windows, constants and the place of layers without feed-forward differ.
CFG_MIXED = (config([par(ff=40), par(heads=6, kv=3, dim=8, vdim=16, window=5, rh=2, rd=12, rv=20, tau=2.0), par(heads=2, kv=1, window=None, tau=16.0, ff=56)]),
             {0: 8, 1: 5, 2: 12})
# nothing a multiple of 8, one head, a window of one token, tau of one
CFG_ODD = (config([par(heads=3, kv=1, dim=6, vdim=10, scale=0.5, window=1, rh=1, rd=5, rv=7, tau=1.0), par(heads=1, kv=1, dim=9, vdim=3, window=4, rh=5, rd=3, rv=9, tau=3.5, ff=21),
                   par(heads=3, kv=3, dim=11, vdim=5, window=30, rh=2, rd=7, rv=5, tau=0.5, ff=17)], width=36, vocab=33, eps=1e-3, escale=0.6, positions=131, cap=3.0),
           {0: 3, 1: 1, 2: 7})
# sizes that the tensor-core kernels take, on both sides of 64 and of one 16-row tile of heads
CFG_WIDE = (config([par(heads=8, kv=2, dim=64, vdim=32, scale=0.125, window=37, rh=2, rd=32, rv=64, ff=96), par(heads=20, kv=5, dim=32, vdim=72, scale=0.2, window=None, rh=4, rd=16, rv=40, ff=64),
                    par(heads=16, kv=16, dim=24, vdim=16, window=50, rh=1, rd=64, rv=32), par(heads=16, kv=1, dim=96, vdim=112, scale=0.1, window=21, rh=2, rd=48, rv=24)],
                   width=128, vocab=150, escale=2.5), {0: 16, 1: 24, 2: 8, 3: 32})
CONFIGS = {"mixed": CFG_MIXED, "odd": CFG_ODD, "wide": CFG_WIDE}


def make_weights(cs, seed):
    """name -> float32 array whose values are exactly representable in bfloat16 (so both engine dtypes hold the same model)."""
    return {k: v.numpy() for k, v in O.random_weights(cs[0], seed, cs[1]).items()}


def build(cfg, weights, dtype="float32", max_tokens=256, slots=4, page_size=4, max_step_tokens=64, cls=None):
    from wf_bitnet import registry
    cls = cls or registry.resolve(cfg)
    model = cls(cfg, dtype=dtype, max_tokens=max_tokens, slots=slots, page_size=page_size, max_step_tokens=max_step_tokens,
                shapes={k: tuple(v.shape) for k, v in weights.items()})
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
    """float32: every row within tolerance.  bfloat16: a position where the random model happens to be ill-conditioned (two keys that
    nearly tie under a sharp softmax, a mixer output whose norm divides by next to nothing) multiplies the rounding below it; such
    positions are few, so four rows in five must be within tolerance, the typical row well within it, and none far off."""
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
    """one part of one layer on given rows, in portions, through the cache and state of one slot"""
    s = m.admit()
    out, a = [], 0
    for c in cuts:
        out.append(m.engine.run_part(layer, part, [s], [c], rows[a:a + c]))
        a += c
    m.release(s)
    return np.concatenate(out)


def oracle_mixer(cfg, w, li, rows):
    return O.pair(torch.from_numpy(rows).double(), t64(w), f"l{li}.mix.", cfg["layers"][li]["mixer"], cfg["norm"]["eps"]).numpy()


def only(w, li, half):
    """the same weights with the other half of layer li's pair silenced by its output norm"""
    w = dict(w)
    other = f"l{li}.mix.{'right' if half == 'left' else 'left'}.out"
    w[other] = np.zeros_like(w[other])
    return w


# ---------------------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixers_alone_whole_and_in_portions(name, dtype):
    """Every layer's pair, and each half of it alone, on random rows: as one portion, in portions of 1 / 2 / 3 / ... tokens through cache
    and state, and token by token."""
    cfg = CONFIGS[name][0]
    full = make_weights(CONFIGS[name], 11)
    n = 45
    for half in (None, "left", "right"):
        w = full
        if half:
            for li in range(len(cfg["layers"])):
                w = only(w, li, half)
        m = build(cfg, w, dtype, max_tokens=512)
        for li in range(len(cfg["layers"])):
            rows = _rows(n, cfg["width"], 20 + li)
            want = oracle_mixer(cfg, w, li, rows)
            for cuts in ([n], [1, 2, 3, 5, 7, 2, 11, 14], [1] * n):
                assert_close(part_alone(m, li, 2, rows, cuts), want, dtype, (name, half, li, cuts[:3]))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_feed_forward_and_norm_alone(dtype):
    for width in (40, 2600):                       # rows that stay in registers, and longer ones
        cfg = config([par(ff=52)], width=width, vocab=40)
        w = make_weights((cfg, {}), 41)
        m = build(cfg, w, dtype, max_step_tokens=256)
        tw = t64(w)
        for n in (1, 7, 150):
            rows = _rows(n, width, 42 + n, 2.0) + 3.0     # a mean that an RMS norm would keep
            h = torch.from_numpy(rows).double()
            assert_close(part_alone(m, 0, 0, rows, [n]), O.layer_norm(h, tw["l0.norm1"], tw["l0.norm1.b"], cfg["norm"]["eps"]).numpy(), "float32", ("norm", width, n))
            assert_close(part_alone(m, 0, 3, bf16_exact(rows), [n]), O.dense_ff(torch.from_numpy(bf16_exact(rows)).double(), tw, "l0.mlp.").numpy(), dtype, ("ff", width, n))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,ff", [(40, 28), (40, None), (38, 28), (1100, 16), (4200, 16), (4201, None), (8300, 16)])
def test_one_layer_gates_both_branches(dtype, width, ff):
    """The stream after a single layer of a one-layer model: gates, pair norms and the sum in one kernel, with and without a feed-forward,
    at widths whose rows fit in registers and beyond, aligned and not.  Opening or closing either gate moves the oracle."""
    cfg = config([par(ff=ff)], width=width, vocab=30)
    w = make_weights((cfg, {}), 45)
    toks = tokens_for(cfg, 12, 46)
    streams = []
    want = oracle_logits(cfg, w, toks, streams)
    for g in ("rg1.b", "rg2.b") if ff else ("rg1.b",):
        other = dict(w); other["l0." + g] = w["l0." + g] + 2
        moved = []
        oracle_logits(cfg, other, toks, moved)
        assert rel_err(moved[0].numpy(), streams[0].numpy()).min() > 2e-3
    m = build(cfg, w, dtype)
    for cuts in ([12], [5] + [1] * 7):
        s, a = m.admit(), 0
        for c in cuts:
            out, tap = m.engine.step_with_layer_tap([s], [c], toks[a:a + c], list(range(c)))
            assert_close(tap[0], streams[0].numpy()[a:a + c], dtype, ("stream", cuts[:2], a), 0.5)
            assert_close(out, want[a:a + c], dtype, ("logits", cuts[:2], a))
            a += c
        m.release(s)
    m.close()


# ------------------------------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_decode_and_portions_agree_with_the_oracle(name, dtype):
    cfg = CONFIGS[name][0]
    w = make_weights(CONFIGS[name], 51)
    m = build(cfg, w, dtype, max_tokens=512)
    n = 61
    toks = tokens_for(cfg, n, 52)
    want = oracle_logits(cfg, w, toks)
    for cuts in ([n], [1] * n, [40] + [1] * 21, [2, 2, 3, 2, 5, 7, 11, 2, 13, 14], [17, 1, 1, 19, 1, 22]):
        assert_close(run_alone(m, toks, cuts), want, dtype, (name, cuts[:4]), 1.5)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_streams_and_first_positions(dtype):
    """Prompts of one to five tokens (shorter than every window): the stream after every layer and the logits."""
    for name in ("odd", "mixed", "wide"):
        cs = CONFIGS[name]
        cfg, w = cs[0], make_weights(cs, 61)
        m = build(cfg, w, dtype)
        for n in (1, 2, 3, 4, 5):
            toks = tokens_for(cfg, n, 62 + n)
            streams = []
            want = oracle_logits(cfg, w, toks, streams)
            s = m.admit()
            out, tap = m.engine.step_with_layer_tap([s], [n], toks, list(range(n)))
            m.release(s)
            for li, st in enumerate(streams):
                assert_close(tap[li], st.numpy(), dtype, ("stream", name, n, li))
            assert_close(out, want, dtype, ("logits", name, n))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_each_request_alone(dtype):
    """Four unequal requests advance together — portions of some beside single tokens of others, one of them paused for a step — and
    every position equals the oracle of its request alone."""
    for name in ("mixed", "wide"):
        cs = CONFIGS[name]
        cfg, w = cs[0], make_weights(cs, 71)
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
    """Six requests through a pool of 12 pages and 2 slots, a neighbour stepping in between: a slot's recurrent state and a page's rows
    must not leak into the next request."""
    cs = CONFIGS["mixed"]
    cfg, w = cs[0], make_weights(cs, 81)
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


def test_the_position_table_ends_where_it_ends():
    cfg = config([par()], positions=10)
    w = make_weights((cfg, {}), 85)
    m = build(cfg, w)
    toks = tokens_for(cfg, 11, 86)
    s = m.admit()
    got = m.step([s], [10], toks[:10], list(range(10)))
    assert_close(got, oracle_logits(cfg, w, toks[:10]), "float32", "to the last position")
    with pytest.raises(ValueError):
        m.step([s], [1], toks[10:], [0])
    m.release(s)
    s = m.admit()
    with pytest.raises(ValueError):
        m.step([s], [11], toks, [10])
    from wf_bitnet.scheduler import Request, Scheduler
    with pytest.raises(ValueError):
        Scheduler(m).add(Request("r", toks[:5], max_new_tokens=7))
    m.close()


# --------------------------------------------------------------------------------------------- one key that decides, at every edge
def _probe_model(dtype, window, page_size, n, heads=4, kv=2, d=32, sharp=1.2):
    """The attention alone, its keys reading the first half of the input row and its queries the second half through the SAME matrix (the
    same one for every head): a probe row that carries in its second half what a marked row carries in its first meets that key with the
    largest score there is (sharp softmax).  The penalty by distance is small here; the mixture of heads is the random one."""
    W = 64
    cfg = config([par(heads=heads, kv=kv, dim=d, vdim=24, scale=sharp, window=window)], width=W, positions=n + 8)
    pre = "l0.mix.left."
    w = only(make_weights((cfg, {}), 91), 0, "left")
    A = _rows(d, W // 2, 92, 1.0 / np.sqrt(W // 2))
    w[pre + "k"] = np.concatenate([np.concatenate([A, np.zeros_like(A)], 1)] * kv, 0)
    w[pre + "q"] = np.concatenate([np.concatenate([np.zeros_like(A), A], 1)] * heads, 0)
    w[pre + "q.norm"] = np.ones_like(w[pre + "q.norm"]); w[pre + "k.norm"] = np.ones_like(w[pre + "k.norm"])
    w[pre + "r1"] = bf16_exact(w[pre + "r1"] * 0.25)
    return cfg, w, build(cfg, w, dtype, max_tokens=n + 64, page_size=page_size, max_step_tokens=n + 8)


def _edge_rows(n, probe, marked, seed):
    rows = _rows(n, 64, seed)
    rows[probe, 32:] = rows[marked, :32]
    return rows


def _cuts(points, n):
    edges = sorted({p for p in points if 0 < p < n} | {0, n})
    return [b - a for a, b in zip(edges, edges[1:])]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("span,page_size,n,probe_back", [(6, 4, 40, 0), (37, 4, 90, 1), (300, 16, 340, 2), (64, 16, 200, 3), (16, 16, 70, 0), (33, 8, 100, 5)])
def test_a_deciding_key_just_inside_and_just_outside_the_window(dtype, span, page_size, n, probe_back):
    """The marked key sits on the last position the probe still sees or one before it; the probe comes at the end of a prompt, in the
    middle of a portion, as a single decoded token, and after portions cut at the marked key.  The two placements differ by tens of
    percent in the oracle, so a window one token off cannot pass."""
    cfg, w, m = _probe_model(dtype, span, page_size, n)
    probe = n - 1 - probe_back
    first_seen = probe - span + 1
    outs = {}
    for where, marked in (("inside", first_seen), ("outside", first_seen - 1), ("near", probe - 1)):
        rows = _edge_rows(n, probe, marked, 93)
        want = oracle_mixer(cfg, w, 0, rows)
        # what the probe would see with the marked key replaced: does the key decide?
        blind = rows.copy()
        blind[marked] = _rows(1, 64, 94)[0]
        outs[where] = rel_err(oracle_mixer(cfg, w, 0, blind)[probe:probe + 1], want[probe:probe + 1])[0]
        for points in ((), (probe, probe + 1), (marked, marked + 2, probe), (marked + 1, probe)):
            cuts = _cuts(points, n)
            got = part_alone(m, 0, 2, rows, cuts)
            assert_close(got[probe:probe + 1], want[probe:probe + 1], dtype, (span, where, cuts), 2.0)
            if dtype == "float32":                 # in bfloat16 two ordinary keys that nearly tie under the sharp softmax may swap
                assert_close(got, want, dtype, (span, where, cuts, "all"), 2.0)
    assert outs["inside"] > 0.3 and outs["near"] > 0.3 and outs["outside"] == 0.0, outs
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size,n,marked", [(64, 400, 0), (64, 400, 1), (64, 400, 63), (64, 400, 64), (64, 400, 65), (16, 330, 127), (16, 330, 128), (4, 90, 3)])
def test_a_far_key_decides_without_a_window(dtype, page_size, n, marked):
    """One key hundreds of positions back, on both sides of page borders and on the very first positions, is the one the last query
    wants; the probe comes at the end of a prompt, after a cut at the marked key, and as a single decoded token.  A reader blind to
    that position differs by tens of percent."""
    cfg, w, m = _probe_model(dtype, None, page_size, n, sharp=2.5)
    probe = n - 1
    rows = _edge_rows(n, probe, marked, 98)
    want = oracle_mixer(cfg, w, 0, rows)
    blind = rows.copy()
    blind[marked] = _rows(1, 64, 99)[0]
    assert rel_err(oracle_mixer(cfg, w, 0, blind)[probe:], want[probe:]).max() > 0.3
    for points in ((), (probe,), (marked + 1, probe), (marked, marked + 2, n - 3, n - 2, probe)):
        got = part_alone(m, 0, 2, rows, _cuts(points, n))
        assert_close(got[probe:], want[probe:], dtype, (marked, points), 2.0)
        if dtype == "float32":
            assert_close(got, want, dtype, (marked, points, "all"), 2.0)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_penalty_takes_off_far_keys(dtype):
    """Two equal keys, one near and one far: the learned penalty decides between them (left out, the output moves by tens of percent)."""
    n = 80
    cfg, w, m = _probe_model(dtype, None, 16, n, sharp=2.5)
    m.close()
    w["l0.mix.left.r1"] = bf16_exact(np.array([1.5, 0.5, 2.0, 1.0])); w["l0.mix.left.r2"] = bf16_exact(np.array([0.05, 1.0, 0.2, 3.0]))
    rows = _edge_rows(n, n - 1, 2, 101)
    rows[n - 5, :32] = rows[2, :32]
    want = oracle_mixer(cfg, w, 0, rows)
    none = dict(w); none["l0.mix.left.r1"] = np.zeros_like(w["l0.mix.left.r1"])
    assert rel_err(oracle_mixer(cfg, none, 0, rows)[-1:], want[-1:])[0] > 0.1
    m = build(cfg, w, dtype, max_tokens=128, page_size=16, max_step_tokens=128)
    for cuts in ([n], [n - 1, 1], [40, 39, 1]):
        assert_close(part_alone(m, 0, 2, rows, cuts)[-1:], want[-1:], dtype, cuts)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [8, 10])
def test_sinks_take_weight_and_are_not_mixed(dtype, dim):
    """Sinks far above and far below the scores, unequal between heads: they change the heads' shares in the mixture (a single head's output
    would only be scaled, which the output norm takes back).  Sinks that take almost everything must not overflow or vanish either."""
    cfg = config([par(heads=4, kv=2, dim=dim, vdim=8, scale=0.1, window=6)], width=32)
    w = only(make_weights((cfg, {}), 171), 0, "left")
    rows = _rows(24, 32, 172)
    for sinks in ([3.0, -1.0, 1.5, 0.25], [40.0, -200.0, 0.0, 2.0], [8.0, 9.0, 8.5, 7.0]):
        w["l0.mix.left.sink"] = bf16_exact(np.array(sinks))
        want = oracle_mixer(cfg, w, 0, rows)
        none = dict(w); none["l0.mix.left.sink"] = np.full(4, -60.0, dtype=np.float32)
        assert rel_err(oracle_mixer(cfg, none, 0, rows), want).max() > 0.1
        m = build(cfg, w, dtype)
        for cuts in ([24], [1] * 24, [5, 2, 17]):
            assert_close(part_alone(m, 0, 2, rows, cuts), want, dtype, (sinks, cuts[:2]))
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dim", [(6, 3, 16), (8, 8, 16), (6, 3, 7), (12, 1, 8), (18, 6, 24), (32, 4, 16)])
def test_heads_are_mixed_across_groups(dtype, heads, kv, dim):
    """A mixture that sends every head's weights to a head of another key/value head (a cyclic shift by one group plus a little of all):
    rows and columns swapped, or values taken from the source's group, would move the oracle far."""
    cfg = config([par(heads=heads, kv=kv, dim=dim, vdim=dim + dim % 2, scale=0.6, window=25)], width=40)
    w = only(make_weights((cfg, {}), 181), 0, "left")
    T = np.roll(np.eye(heads), heads // kv + 1, 0) + np.random.default_rng(182).standard_normal((heads, heads)) * 0.15
    w["l0.mix.left.talk"] = bf16_exact(T)
    rows = _rows(60, 40, 183)
    want = oracle_mixer(cfg, w, 0, rows)
    turned = dict(w); turned["l0.mix.left.talk"] = np.ascontiguousarray(w["l0.mix.left.talk"].T)
    assert np.median(rel_err(oracle_mixer(cfg, turned, 0, rows)[5:], want[5:])) > 0.2
    m = build(cfg, w, dtype, max_tokens=128)
    for cuts in ([60], [1] * 60, [7, 2, 30, 1, 20]):
        assert_close(part_alone(m, 0, 2, rows, cuts), want, dtype, (heads, kv, cuts[:2]))
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 10])
def test_penalty_and_sinks_without_a_mixture(dtype, dim):
    """The logarithmic penalty and the learned sinks in the attention kernels that do not mix heads: the engine's descriptor without `talk`
    equals the oracle with the identity as the mixture."""
    from wf_bitnet import registry
    cfg = config([par(heads=4, kv=2, dim=dim, vdim=16, window=400)], width=40, positions=400)

    class Unmixed(registry.resolve(cfg)):
        @staticmethod
        def read_config(c, shapes=None):
            r = registry.resolve(cfg).read_config(c, shapes)
            layers = r.native_layers
            def without():
                out = layers()
                out[0].talk = 0
                return out
            r.native_layers = without
            return r

    w = only(make_weights((cfg, {}), 191), 0, "left")
    w["l0.mix.left.talk"] = np.eye(4, dtype=np.float32)
    w["l0.mix.left.sink"] = bf16_exact(np.array([2.0, -1.0, 30.0, 0.5]))
    n = 330
    rows = _rows(n, 40, 192)
    want = oracle_mixer(cfg, w, 0, rows)
    m = build(cfg, w, dtype, max_tokens=4096, page_size=16, max_step_tokens=512, cls=Unmixed)
    assert not any(name.endswith("talk") for name, _, _ in m.engine.expected_tensors())
    for cuts in ([n], [n - 6] + [1] * 6, [100, 2, 228]):
        assert_close(part_alone(m, 0, 2, rows, cuts), want, dtype, cuts[:2])
    m.close()


# ------------------------------------------------------------------------------------------------------- recurrence, long sequences
def test_state_is_carried_over_hundreds_of_tokens():
    """A recurrence made to forget slowly: 300 tokens in seven portions with a neighbour stepping in another slot.  A state that lost its
    first half would move the last outputs by more than a tenth."""
    cfg = config([par(rh=2, rd=16, rv=8, tau=16.0)], width=32)
    w = only(make_weights((cfg, {}), 101), 0, "right")
    w["l0.mix.right.a2.b"] = np.full_like(w["l0.mix.right.a2.b"], 4.0)
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
@pytest.mark.parametrize("rd,rv,bias,tau", [(12, 10, 2.0, 8.0), (40, 24, -3.0, 0.7), (128, 40, 0.0, 16.0)])
def test_long_portions_of_the_recurrence(dtype, rd, rv, bias, tau):
    """Portions of several hundred tokens run the recurrence in parallel chunks whose start states are chained with the products of the
    chunks' decays, one per key row: a long portion after a short one, then a ragged batch of a long, a short and a chunk-sized portion in
    three slots, against the token-by-token oracle.  Decays from almost one to almost zero, unequal between key rows."""
    cfg = config([par(rh=3, rd=rd, rv=rv, tau=tau)], width=32, positions=1024)
    w = only(make_weights((cfg, {0: 6}), 161), 0, "right")
    w["l0.mix.right.a2.b"] = bf16_exact(w["l0.mix.right.a2.b"] * 2 + bias)
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
    """150 decoded tokens on 4-token pages: windows slide over decoded tokens only, positions grow."""
    for name in ("mixed", "wide"):
        cs = CONFIGS[name]
        cfg, w = cs[0], make_weights(cs, 121)
        m = build(cfg, w, dtype, max_tokens=256, page_size=4)
        toks = tokens_for(cfg, 160, 122)
        assert_close(run_alone(m, toks, [10] + [1] * 150), oracle_logits(cfg, w, toks), dtype, ("decode", name), 1.5)
        m.close()


@pytest.mark.parametrize("heads,kv,dim,vdim,window", [(8, 2, 64, 64, None), (20, 5, 128, 128, 700), (16, 16, 64, 128, 300)])
def test_tensor_core_attention_with_key_splits_in_a_ragged_batch(heads, kv, dim, vdim, window):
    """bfloat16, sizes the tensor-core kernels take, contexts long enough that decoding cuts the keys over several blocks: three sequences
    of unequal length, prompts in portions and then decoded together; float32 (the plain kernels) beside it."""
    cfg = config([par(heads=heads, kv=kv, dim=dim, vdim=vdim, scale=dim ** -0.5, window=window, rh=2, rd=8, rv=8)], width=64, vocab=90, positions=700)
    w = make_weights((cfg, {}), 131)
    lens = (650, 300, 41)
    reqs = [tokens_for(cfg, n + 6, 132 + n) for n in lens]
    want = [oracle_logits(cfg, w, r) for r in reqs]
    for dtype in ("bfloat16", "float32"):
        m = build(cfg, w, dtype, max_tokens=1200, page_size=16, max_step_tokens=512)
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
    """1-4 layers with sizes drawn independently of each other"""
    W = rng.choice([24, 40, 72, 96, 136, 200])
    layers, ranks = [], {}
    for i in range(rng.randint(1, 4)):
        G, rep = rng.choice([1, 2, 3, 5]), rng.choice([1, 2, 3, 4, 6])
        d = rng.choice([6, 16, 24, 64, 104, 128, 160])
        layers.append(par(heads=G * rep, kv=G, dim=d, vdim=rng.choice([d, 8, 40, 65, 128]), scale=rng.choice([d ** -0.5, 0.2]), window=rng.choice([None, 1, 2, 7, 16, 50, 120]),
                          rh=rng.choice([1, 2, 5]), rd=rng.choice([4, 16, 33, 72, 160]), rv=rng.choice([4, 24, 40, 136]), tau=rng.choice([0.5, 1.0, 9.0, 16.0]),
                          ff=rng.choice([None, W, rng.randint(8, 3 * W)])))
        ranks[i] = rng.choice([1, 4, 16, 30])
    return config(layers, width=W, vocab=rng.choice([50, 97, 300]), eps=rng.choice([1e-6, 1e-4]), escale=rng.choice([1.0, W ** 0.5, 0.3]), positions=rng.choice([300, 1000]),
                  cap=rng.choice([2.0, 15.0, 50.0])), ranks


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations(seed):
    """Head counts, sizes, windows and constants drawn at random: one prompt whole, prompt + decoded tail, and in random portions, in both
    dtypes."""
    import random
    rng = random.Random(1000 + seed)
    cfg, ranks = _random_config(rng)
    n = rng.choice([3, 17, 64, 130, 290])
    w = make_weights((cfg, ranks), 200 + seed)
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
    cs = CONFIGS["mixed"]
    cfg, w = cs[0], make_weights(cs, 141)
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
    one; `generate` runs the scheduler.  The model class comes from config.json, the inner sizes from the checkpoint's shapes."""
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    cs = CONFIGS["mixed"]
    cfg, w = cs[0], make_weights(cs, 151)
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
