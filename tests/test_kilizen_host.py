"""Kilizen without a device: the configuration reader (every size and constant from config.json), the registry, and checks of the oracle
itself."""
import copy
import math

import numpy as np
import pytest
import torch

import kilizen_oracle as O
from test_gpu_kilizen import CONFIGS, _rows, config, ffd, full, make_weights, mem, moe, rel_err, rope, t64, win


def _native(cfg):
    from sglang.srt.models.kilizen import KilizenConfig
    c = KilizenConfig.from_dict(cfg)
    return c, c.native_layers()


def test_registry_resolves_the_architecture():
    from wf_bitnet import registry
    assert registry.resolve({"architecture": "Kilizen"}).__name__ == "KilizenForCausalLM"
    assert registry.resolve({"architectures": ["KilizenForCausalLM"]}).__name__ == "KilizenForCausalLM"


def test_config_reader_takes_every_size_and_constant():
    from wf_bitnet import _lib
    for cfg in CONFIGS.values():
        c, nat = _native(cfg)
        assert len(nat) == len(cfg["layers"])
        for L, s in zip(cfg["layers"], nat):
            m, f = L["mixer"], L["mlp"]
            assert (s.heads, s.dim, s.vdim) == (m["heads"], m["dim"], m["vdim"])
            if L["type"] == "mlstm":
                assert s.type == _lib.WF_SEQ_MLSTM and s.gate_cap == pytest.approx(m["gate_cap"])
            else:
                one = L["type"] == "attention"
                assert (s.type, s.kv_heads, s.sink, s.rope_dims, s.rope_interleaved, s.head_gate) == (_lib.WF_SEQ_GQA_ATTENTION, m["kv_heads"], 2, m["rot"]["dims"], 0, 0)
                assert s.scale == pytest.approx(m["scale"]) and s.rope_base == pytest.approx(m["rot"]["base"])
                assert (s.v_is_k, s.proj_bias) == ((2, 0) if one else (0, 1))
                assert s.qk_norm == (_lib.WF_SEQ_QKNORM_HEAD if one else _lib.WF_SEQ_QKNORM_FULL)
                assert (s.window, s.keep_first) == ((m["mask"]["size"], m["mask"]["keep_first"]) if one else (1 << 30, 0))
                sc = m["rot"].get("scaling")
                assert (s.rope_factor, s.rope_orig, s.rope_fast, s.rope_slow) == pytest.approx((sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else (0, 0, 0, 0))
            if not f:
                assert s.has_ff == _lib.WF_SEQ_FF_NONE
            elif f["kind"] == "dense":
                assert (s.has_ff, s.ff, s.ff_act) == (_lib.WF_SEQ_FF_DENSE, f["ff"], _lib.WF_SEQ_ACT_GELU_ERF)
            else:
                assert (s.has_ff, s.ff, s.ff_act, s.experts, s.top) == (_lib.WF_SEQ_FF_ROUTED, f["expert"]["ff"], _lib.WF_SEQ_ACT_RELU2, f["router"]["experts"], f["router"]["top"])
                assert (s.shared_ff, s.shared_plain, s.no_correction, s.router_norm, s.router_act) == (f.get("shared", {"ff": 0})["ff"], 1, 1, 1, 0)
        nc = _lib.SeqConfig()
        c.fill_native(nc)
        assert (nc.block_form, nc.norm_kind, nc.canon_taps, nc.tied_head) == (_lib.WF_SEQ_BLOCK_SANDWICH, _lib.WF_SEQ_NORM_DYN_TANH, 0, 0)
        assert (nc.loop_start, nc.loop_stop, nc.loop_times) == tuple(cfg["loop"][k] for k in ("start", "stop", "times"))
    bare = full()
    bare["mixer"].pop("rot")
    assert _native(config([bare]))[1][0].rope_dims == 0
    free = win()
    free["mixer"].pop("mask")
    assert _native(config([free]))[1][0].window >= 1 << 30


def test_config_reader_rejects_what_it_cannot_serve():
    for bad in (config([]), config([dict(mem(), type="convolution")]), config([mem(mlp={"kind": "gated", "ff": 8})]), config([mem()], loop=(0, 2, 2)), config([mem(), mem()], loop=(1, 1, 2))):
        with pytest.raises(ValueError):
            _native(bad)
    p = win()
    p["mixer"]["vdim"] = 24                       # values that are the keys cannot have a size of their own
    with pytest.raises(ValueError):
        _native(config([p]))


def test_oracle_pieces():
    w = {"n": torch.tensor([2.0, 3.0]), "n.b": torch.tensor([0.5, -1.0]), "n.alpha": torch.tensor(0.5)}
    x = torch.tensor([[1.0, -4.0]])
    assert torch.allclose(O.dyn_tanh(x, w, "n"), torch.tensor([[2 * math.tanh(0.5) + 0.5, -3 * math.tanh(2.0) - 1.0]]))
    assert O.gelu_exact(torch.tensor(1.0, dtype=torch.float64)) == pytest.approx(0.8413447460685429)
    seen = O.visible(8, {"size": 3, "keep_first": 2})
    assert seen[7].tolist() == [True, True, False, False, False, True, True, True] and seen[1].tolist() == [True, True] + [False] * 6
    assert torch.equal(O.visible(5, None), torch.ones(5, 5).tril().bool())
    p = O.sink_softmax(torch.tensor([[0.0, -math.inf, 0.0]]), torch.tensor(0.0))
    assert torch.allclose(p, torch.tensor([[1 / 3, 0.0, 1 / 3]]))
    idx, wt = O.choose(torch.tensor([[0.0, 2.0, 1.0, -5.0]], dtype=torch.float64), 2)
    assert idx.tolist() == [[1, 2]] and wt[0, 0] == pytest.approx(1 / (1 + math.exp(-1.0)))
    f, mag = O.turn_rates(rope(8, 100.0, (4.0, 32, 8.0, 1.0)))
    plain, one = O.turn_rates(rope(8, 100.0))
    assert one == 1.0 and mag == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 4.0) and all(plain[i] / 4 <= f[i] <= plain[i] for i in range(4))
    x = torch.zeros(1, 1, 5, dtype=torch.float64)
    x[0, 0, 0] = 1.0                              # entry 0 turns with entry 2, entry 4 stays
    y = O.rotate_half(x, torch.tensor([3]), rope(4, 10.0))[0, 0]
    assert y.tolist() == pytest.approx([math.cos(3.0), 0.0, math.sin(3.0), 0.0, 0.0])


def test_layer_runs_of_a_loop():
    three = [mem(), mem(), mem()]
    assert [i for i, _ in O.layer_runs(config(three, loop=(1, 3, 3)))] == [0, 1, 2, 1, 2, 1, 2]
    assert [k for k, (_, again) in enumerate(O.layer_runs(config(three, loop=(1, 3, 3)))) if again] == [3, 5]
    assert O.layer_runs(config(three, loop=(0, 1, 2))) == [(0, False), (0, True), (1, False), (2, False)]
    assert O.layer_runs(config(three)) == [(0, False), (1, False), (2, False)]


def test_oracle_is_sensitive_to_every_mechanism():
    """Each constant and each special rule moves the oracle's output: a product path that ignored one of them could not agree with it."""
    rows = torch.from_numpy(_rows(40, 48, 5)).double()

    def moved(layer, change):
        cfg = config([layer])
        w = t64(make_weights(cfg, 7))
        base = O.MIXERS[layer["type"]](rows, w, "l0.mix.", layer["mixer"], 2e-5).numpy()
        other, w2 = copy.deepcopy(layer["mixer"]), dict(w)
        change(other, w2)
        return rel_err(O.MIXERS[layer["type"]](rows, w2, "l0.mix.", other, 2e-5).numpy(), base).max()

    A, B, M = win(), full(), mem()
    assert moved(A, lambda m, w: m["mask"].update(size=8)) > 1e-2                 # the window, by one token
    assert moved(A, lambda m, w: m["mask"].update(keep_first=2)) > 1e-2           # the kept positions, by one
    assert moved(A, lambda m, w: m["rot"].pop("scaling")) > 1e-2
    for L in (A, B):
        assert moved(L, lambda m, w: m["rot"].update(base=200.0)) > 1e-3
        assert moved(L, lambda m, w: m.update(scale=0.4)) > 1e-2
        assert moved(L, lambda m, w: w.update({"l0.mix.sink": w["l0.mix.sink"] + 1})) > 1e-2
        assert moved(L, lambda m, w: w.update({"l0.mix.k.norm": w["l0.mix.k.norm"] * 0 + 1})) > 1e-3
    for b in ("q.b", "k.b", "v.b", "o.b"):
        assert moved(B, lambda m, w: w.update({"l0.mix." + b: w["l0.mix." + b] * 0})) > 1e-2
    assert moved(M, lambda m, w: m.update(gate_cap=1.0)) > 1e-2
    assert moved(M, lambda m, w: w.update({"l0.mix.f.b": w["l0.mix.f.b"] - 3})) > 1e-2
    assert moved(M, lambda m, w: w.update({"l0.mix.i.b": w["l0.mix.i.b"] + 1})) > 1e-4
    f = moe()
    w = t64(make_weights(config([mem(mlp=f)]), 8))
    y = O.routed_ff(rows, w, "l0.mlp.", f)
    assert rel_err(O.routed_ff(rows, w, "l0.mlp.", moe(top=3)).numpy(), y.numpy()).max() > 1e-2
    assert rel_err(O.routed_ff(rows, w, "l0.mlp.", moe(shared=0)).numpy(), y.numpy()).max() > 1e-2
    assert rel_err(O.dense_ff(rows, {"up": w["l0.mlp.e0.up"], "down": w["l0.mlp.e0.down"]}, "").numpy(), O.expert(rows, w, "l0.mlp.e0.").numpy()).max() > 1e-2


def test_prefixes_agree():
    """Causality of the whole oracle: the first logits do not change when tokens follow."""
    for cfg in CONFIGS.values():
        w = t64(make_weights(cfg, 9))
        toks = np.random.default_rng(1).integers(0, cfg["vocab"], 20).tolist()
        assert np.allclose(O.forward(cfg, w, toks)[:11].numpy(), O.forward(cfg, w, toks[:11]).numpy(), atol=1e-9)
