"""Fuvavik without a device: the configuration reader (every size and constant from config.json or the checkpoint's tensor shapes), the
registry, the scheduler's position limit, and checks of the oracle itself."""
import numpy as np
import pytest
import torch

import fuvavik_oracle as O
from test_gpu_fuvavik import CONFIGS, _rows, config, make_weights, par, rel_err, t64


def _native(cs, seed=1):
    from sglang.srt.models.fuvavik import FuvavikConfig
    c = FuvavikConfig.from_dict(cs[0], {k: v.shape for k, v in make_weights(cs, seed).items()})
    return c, c.native_layers()


def test_registry_resolves_the_architecture():
    from wf_bitnet import registry
    assert registry.resolve({"architecture": "Fuvavik"}).__name__ == "FuvavikForCausalLM"
    assert registry.resolve({"architectures": ["FuvavikForCausalLM"]}).reads_shapes


def test_config_reader_takes_every_size_from_config_and_shapes():
    from wf_bitnet import _lib
    for cs in CONFIGS.values():
        cfg = cs[0]
        c, nat = _native(cs)
        layers = cfg["layers"]
        assert len(nat) == 2 * len(layers)
        for i, L in enumerate(layers):
            a, r, s, x = L["mixer"]["left"], L["mixer"]["right"], nat[i], nat[nat[i].pair]
            assert s.pair == len(layers) + i and (s.pair_norm, s.mix_scale, s.pair_scale) == (1, 0.5, 0.5)
            assert (s.type, s.heads, s.kv_heads, s.dim, s.vdim) == (_lib.WF_SEQ_GQA_ATTENTION, a["heads"], a["kv_heads"], a["dim"], a["vdim"])
            assert s.window == a["mask"]["size"] if "mask" in a else s.window >= 1 << 30
            assert s.scale == pytest.approx(a["scale"]) and (s.dist_log, s.sink, s.talk, s.qk_norm) == (1, 2, 1, _lib.WF_SEQ_QKNORM_FULL)
            assert (s.proj_bias, s.head_gate, s.rope_dims, s.chunk, s.rel_rows, s.v_is_k) == (0, 0, 0, 0, 0, 0) and s.softcap == 0.0 and s.dist_exp == 0.0
            assert (x.type, x.heads, x.dim, x.vdim, x.decay_rank) == (_lib.WF_SEQ_GLA, r["heads"], r["dim"], r["vdim"], cs[1][i]) and x.decay_tau == pytest.approx(r["tau"])
            if L["mlp"]:
                assert (s.has_ff, s.ff, s.ff_act) == (_lib.WF_SEQ_FF_DENSE, L["mlp"]["ff"], _lib.WF_SEQ_ACT_GELU_TANH)
            else:
                assert s.has_ff == _lib.WF_SEQ_FF_NONE
        nc = _lib.SeqConfig()
        c.fill_native(nc)
        assert (nc.block_form, nc.layer_norm, nc.one_norm, nc.branch_gates, nc.tied_head, nc.pos_embed) == (_lib.WF_SEQ_BLOCK_PARALLEL, 1, 1, 1, 1, 2)
        assert nc.max_positions == cfg["max_positions"] and nc.logit_softcap == pytest.approx(cfg["logit_softcap"]) and nc.embed_scale == pytest.approx(cfg["embedding"]["scale"])


def test_config_reader_rejects_what_it_cannot_serve():
    from sglang.srt.models.fuvavik import FuvavikConfig
    cs = CONFIGS["mixed"]
    cfg, shapes = cs[0], {k: v.shape for k, v in make_weights(cs, 1).items()}
    for bad in (dict(cfg, layers=[dict(cfg["layers"][0], type="attention")]), dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "moe", "ff": 8})])):
        with pytest.raises(ValueError):
            FuvavikConfig.from_dict(bad, shapes).native_layers()
    with pytest.raises(ValueError):
        FuvavikConfig.from_dict(cfg, {}).native_layers()             # the decay projection's inner size is in the shapes only
    with pytest.raises(ValueError):
        FuvavikConfig.from_dict(dict(cfg, layers=[]), shapes)
    short = {k: v for k, v in cfg.items() if k != "max_positions"}
    assert FuvavikConfig.from_dict(short, shapes).max_positions == cfg["max_positions"]      # the table's rows say it too
    with pytest.raises(ValueError):
        FuvavikConfig.from_dict(short, {})


def test_scheduler_refuses_requests_beyond_the_position_table():
    from wf_bitnet.scheduler import Request, Scheduler

    class Model:
        max_step_tokens, max_positions = 64, 20
    s = Scheduler(Model())
    s.add(Request("fits", [1] * 15, max_new_tokens=6))               # the sixth drawn token is not fed back: 20 positions
    with pytest.raises(ValueError):
        s.add(Request("long", [1] * 15, max_new_tokens=7))


def test_oracle_is_sensitive_to_every_mechanism():
    """Each constant and each special rule moves the oracle's output: a product path that ignored one of them could not agree with it."""
    cfg = config([par(heads=4, kv=2, window=9, ff=40), par(heads=4, kv=2, window=30)], positions=60, cap=4.0)
    w = t64(make_weights((cfg, {0: 8, 1: 8}), 7))
    toks = np.random.default_rng(8).integers(0, cfg["vocab"], 40).tolist()
    base = O.forward(cfg, w, toks).numpy()

    def moved(least, **tensors):
        w2 = dict(w)
        for name, f in tensors.items():
            n = name.replace("__", ".")
            w2[n] = f(w[n])
        return rel_err(O.forward(cfg, w2, toks).numpy(), base).max() > least

    zero, one = torch.zeros_like, torch.ones_like
    assert moved(1e-2, pos=zero) and moved(1e-2, final__norm__b=zero) and moved(1e-2, l0__norm1__b=zero)
    assert moved(1e-2, l0__mix__left__r1=zero) and moved(1e-3, l0__mix__left__r2=lambda t: t * 2) and moved(1e-3, l0__mix__left__sink=lambda t: t - 30)
    assert moved(1e-2, l0__mix__left__talk=lambda t: t.T.contiguous()) and moved(1e-3, l0__mix__left__q__norm=one) and moved(1e-3, l0__mix__left__k__norm=one)
    assert moved(1e-2, l1__mix__left__out=one) and moved(1e-2, l1__mix__right__out=one) and moved(1e-3, l0__mix__right__norm=one)
    assert moved(1e-3, l0__mix__right__a2__b=lambda t: t - 1) and moved(1e-2, l0__rg1__b=lambda t: t + 1) and moved(1e-2, l0__rg2__b=lambda t: t + 1)

    def reconfigured(edit):
        import copy
        c = copy.deepcopy(cfg)
        edit(c)
        return rel_err(O.forward(c, w, toks).numpy(), base).max()

    assert reconfigured(lambda c: c.update(logit_softcap=8.0)) > 1e-2
    assert reconfigured(lambda c: c["embedding"].update(scale=1.5)) > 1e-2
    assert reconfigured(lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=8)) > 1e-3
    assert reconfigured(lambda c: c["layers"][0]["mixer"]["left"].pop("mask")) > 1e-3
    assert reconfigured(lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.4)) > 1e-3
    assert reconfigured(lambda c: c["layers"][0]["mixer"]["right"].update(tau=4.0)) > 1e-3


def test_oracle_pieces():
    """Closed forms: the penalty, a softmax whose sink takes a known share, a layer norm that forgets a shift, the recurrence against its sum."""
    assert O.log_penalty(torch.tensor(4.0), torch.tensor(2.0), torch.tensor(0.5)).item() == pytest.approx(2 * np.log(3.0))
    p = O.softmax_with_sink(torch.tensor([0.0, float("-inf"), 0.0]).double(), torch.tensor(np.log(2.0)))
    assert p.tolist() == pytest.approx([0.25, 0.0, 0.25])
    x = torch.from_numpy(_rows(3, 20, 1)).double()
    g, b = torch.full((20,), 2.0).double(), torch.full((20,), 0.5).double()
    assert torch.allclose(O.layer_norm(x, g, b, 1e-6), O.layer_norm(x + 7, g, b, 1e-6), atol=1e-9)
    assert O.layer_norm(x, g, b, 0.0).std(-1, unbiased=False).tolist() == pytest.approx([2.0] * 3)
    cfg = config([par(rh=1, rd=4, rv=3, tau=5.0)], width=16)
    w = t64(make_weights((cfg, {0: 2}), 9))
    p_, m, h = "l0.mix.right.", cfg["layers"][0]["mixer"]["right"], torch.from_numpy(_rows(12, 16, 10)).double()
    a = O.channel_decay(h, w, p_, 5.0)
    z = (h @ w[p_ + "a1"].T) @ w[p_ + "a2"].T + w[p_ + "a2.b"]
    assert torch.allclose(a, torch.sigmoid(z) ** 0.2)
    q, k, v = (h @ w[p_ + n].T for n in ("q", "k", "v"))
    o = torch.stack([sum((q[t] * k[j] * a[j + 1:t + 1].prod(0)).sum() * v[j] for j in range(t + 1)) for t in range(12)]) / 2.0
    want = (O.unit_rms(o, 2e-5) * w[p_ + "norm"] * O.silu(h @ w[p_ + "g"].T)) @ w[p_ + "o"].T
    assert rel_err(O.gated_linear(h, w, p_, m, 2e-5).numpy(), want.numpy()).max() < 1e-9
