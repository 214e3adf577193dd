"""Kilizen: a decoder-only stack whose sublayers sit between two element-wise norms tanh(alpha x) w + b, x <- x + n1b(mixer(n1(x))), then
x <- x + n2b(ff(n2(x))).  A range of layers can run several times in a row with the same weights; every pass keeps its own cache and state,
and the embedding is added to the stream before each pass but the first.  Three kinds of mixer:

  'attention'    grouped-query attention without a value projection: the values are the keys as projected, before their RMS norm (per head,
                 one shared weight vector) and rotation (the first rot.dims entries in half-split pairs, frequencies interpolated where the
                 configuration says so); a sliding window beside a few first positions that stay visible; a learned per-head sink;
  'attention_2'  causal grouped-query attention with biased projections, RMS norm over the whole query / key projection, half-split
                 rotation, a learned per-head sink;
  'mlstm'        a matrix memory with exponential input gate, sigmoid forget gate (both capped by a tanh) and a running maximum of the log
                 gates.
The feed-forward is dense, down(gelu(up h)) with the erf form of gelu, or routed: experts down(relu(up h)^2), the `top` largest router logits
weighted by a softmax over themselves, and a shared expert added for every token.

This module is the model's configuration reader and its binding to the native engine (libwf_seq.so); it computes nothing itself.
config.json keys read here: architecture, vocab, width, norm.eps, loop.{start, stop, times}, layers[].{type, mixer.{heads, kv_heads, dim,
vdim, scale, mask.{size, keep_first}, rot.{dims, base, scaling.{factor, original, fast, slow}}, gate_cap}, mlp.{kind, ff, router.{experts,
top}, expert.ff, shared.ff}}.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List

from wf_bitnet import _lib
from wf_bitnet._lib import SeqConfig, SeqLayer
from wf_bitnet.seq_model import SeqCausalLM

NO_WINDOW = 1 << 30


@dataclass
class KilizenConfig:
    vocab: int
    width: int
    eps: float
    layers: List[dict] = field(default_factory=list)
    loop: Dict[str, int] = field(default_factory=dict)

    @staticmethod
    def from_dict(cfg: Dict) -> "KilizenConfig":
        out = KilizenConfig(vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), layers=list(cfg["layers"]),
                            loop={k: int(v) for k, v in (cfg.get("loop") or {}).items()})
        if not out.layers:
            raise ValueError("config: 'layers' is empty")
        if out.loop and not (0 <= out.loop["start"] < out.loop["stop"] <= len(out.layers) and out.loop["times"] >= 1):
            raise ValueError(f"config: loop {out.loop} does not name layers of {len(out.layers)}")
        return out

    def fill_native(self, nc: SeqConfig) -> None:
        nc.block_form, nc.norm_kind = _lib.WF_SEQ_BLOCK_SANDWICH, _lib.WF_SEQ_NORM_DYN_TANH
        nc.canon_taps, nc.tied_head = 0, 0
        if self.loop:
            nc.loop_start, nc.loop_stop, nc.loop_times = self.loop["start"], self.loop["stop"], self.loop["times"]

    @staticmethod
    def _attention(m: Dict) -> SeqLayer:
        """What both kinds of attention share."""
        s = SeqLayer()
        s.type = _lib.WF_SEQ_GQA_ATTENTION
        s.heads, s.dim = int(m["heads"]), int(m["dim"])
        s.vdim = int(m.get("vdim", s.dim))
        s.kv_heads = int(m.get("kv_heads", s.heads))
        s.scale = float(m["scale"])
        mask = m.get("mask") or {}
        s.window = int(mask["size"]) if "size" in mask else NO_WINDOW
        s.keep_first = int(mask.get("keep_first", 0))
        s.sink = 2
        rot = m.get("rot") or {}
        s.rope_dims, s.rope_base = int(rot.get("dims", 0)), float(rot.get("base", 10000.0))
        sc = rot.get("scaling")
        if sc:
            s.rope_factor, s.rope_orig = float(sc["factor"]), float(sc["original"])
            s.rope_fast, s.rope_slow = float(sc["fast"]), float(sc["slow"])
        return s

    @classmethod
    def _window_attention(cls, m: Dict, what: str) -> SeqLayer:
        s = cls._attention(m)
        if s.vdim != s.dim:
            raise ValueError(f"config: {what}: the values are the keys, so vdim ({s.vdim}) must equal dim ({s.dim})")
        s.v_is_k, s.qk_norm = 2, _lib.WF_SEQ_QKNORM_HEAD
        return s

    @classmethod
    def _full_attention(cls, m: Dict) -> SeqLayer:
        s = cls._attention(m)
        s.proj_bias, s.qk_norm = 1, _lib.WF_SEQ_QKNORM_FULL
        return s

    @staticmethod
    def _matrix_memory(m: Dict) -> SeqLayer:
        s = SeqLayer()
        s.type = _lib.WF_SEQ_MLSTM
        s.heads, s.dim, s.vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        s.gate_cap = float(m["gate_cap"])
        return s

    @staticmethod
    def _feed_forward(s: SeqLayer, f: Dict, what: str) -> None:
        if f is None:
            s.has_ff = _lib.WF_SEQ_FF_NONE
        elif f.get("kind") == "dense":
            s.has_ff, s.ff_act, s.ff = _lib.WF_SEQ_FF_DENSE, _lib.WF_SEQ_ACT_GELU_ERF, int(f["ff"])
        elif f.get("kind") == "moe":
            s.has_ff, s.ff_act, s.ff = _lib.WF_SEQ_FF_ROUTED, _lib.WF_SEQ_ACT_RELU2, int(f["expert"]["ff"])
            s.experts, s.top = int(f["router"]["experts"]), int(f["router"]["top"])
            s.groups, s.keep, s.group_top = 1, 1, 1
            # a softmax over all logits, divided by the chosen ones' sum, is the softmax over the chosen logits
            s.router_act, s.router_norm, s.no_correction = 0, 1, 1
            s.shared_ff = int(f["shared"]["ff"]) if f.get("shared") else 0
            s.shared_plain = 1
        else:
            raise ValueError(f"config: {what} has unknown feed-forward kind {f.get('kind')!r}")

    def native_layers(self) -> List[SeqLayer]:
        out = []
        for i, L in enumerate(self.layers):
            m, kind, what = L["mixer"], L["type"], f"layer {i}"
            if kind == "attention":
                s = self._window_attention(m, what)
            elif kind == "attention_2":
                s = self._full_attention(m)
            elif kind == "mlstm":
                s = self._matrix_memory(m)
            else:
                raise ValueError(f"config: {what} has unknown mixer type {kind!r}")
            self._feed_forward(s, L.get("mlp"), what)
            out.append(s)
        return out


class KilizenForCausalLM(SeqCausalLM):
    """Model class of the registry (weights, engine and step interface: wf_bitnet.seq_model.SeqCausalLM)."""

    architecture_names = ("Kilizen", "KilizenForCausalLM")

    @staticmethod
    def read_config(config: Dict) -> KilizenConfig:
        return KilizenConfig.from_dict(config)


EntryClass = KilizenForCausalLM
