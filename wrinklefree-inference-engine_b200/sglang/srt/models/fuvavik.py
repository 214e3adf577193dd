"""Fuvavik: a decoder-only stack whose layers have ONE layer norm (mean taken off, weight and bias) whose output h both branches read; each
branch's result is multiplied element by element by a sigmoid gate computed from h: x <- x + s(R1 h + b1) * mixer(h) + s(R2 h + b2) * ff(h).
The stream starts as the scaled embedding plus a learned vector per position; the logits are products with the unscaled embedding table,
capped by a tanh.  One kind of mixer:

  'parallel'   two mixers side by side on the same input, each output RMS-normed over the width with a weight vector, half the sum of both:
               left   grouped-query attention without rotation: RMS norm over the whole query / key projection, a sliding window, the
                      distance penalty r1 ln(1 + r2 distance) with learned numbers per head, a learned sink per head in the softmax
                      denominator, and the heads' weights mixed by a learned matrix before they meet the values;
               right  gated linear attention: a matrix state per head whose key rows decay each by sigmoid(z)^(1 / tau), z from a
                      two-matrix projection with bias; per-head output norm, silu gate.

The feed-forward is a gelu-gated (tanh form) dense unit, or absent.

This module is the model's configuration reader and its binding to the native engine (libwf_seq.so); it computes nothing itself.
config.json keys read here: architecture, vocab, width, embedding.scale, norm.eps, max_positions, logit_softcap, layers[].{type,
mlp.{kind, ff}, mixer.left.{heads, kv_heads, dim, vdim, scale, mask.size}, mixer.right.{heads, dim, vdim, tau}}.  The inner size of the
two-matrix decay projection is read from the checkpoint's tensor shapes (`mix.right.a1`).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

from wf_bitnet import _lib
from wf_bitnet._lib import SeqConfig, SeqLayer
from wf_bitnet.seq_model import SeqCausalLM

NO_WINDOW = 1 << 30


@dataclass
class FuvavikConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    max_positions: int
    logit_softcap: float
    layers: List[dict] = field(default_factory=list)
    shapes: Dict[str, tuple] = field(default_factory=dict)      # tensor name -> shape, from the checkpoint header

    @staticmethod
    def from_dict(cfg: Dict, shapes: Optional[Dict[str, tuple]] = None) -> "FuvavikConfig":
        shapes = dict(shapes or {})
        positions = cfg.get("max_positions", shapes["pos"][0] if "pos" in shapes else None)
        if positions is None:
            raise ValueError("config: 'max_positions' is missing and no tensor shapes name the position table's rows")
        out = FuvavikConfig(vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]),
                            max_positions=int(positions), logit_softcap=float(cfg.get("logit_softcap") or 0.0), layers=list(cfg["layers"]), shapes=shapes)
        if not out.layers:
            raise ValueError("config: 'layers' is empty")
        return out

    def fill_native(self, nc: SeqConfig) -> None:
        nc.block_form = _lib.WF_SEQ_BLOCK_PARALLEL
        nc.norm_weights, nc.tied_head = 1, 1
        nc.layer_norm, nc.one_norm, nc.branch_gates = 1, 1, 1
        nc.embed_scale = self.embed_scale
        nc.pos_embed, nc.max_positions = 2, self.max_positions
        nc.logit_softcap = self.logit_softcap

    def _rows(self, name: str, what: str) -> int:
        if name not in self.shapes:
            raise ValueError(f"config: {what} is the row count of tensor {name!r}; pass the checkpoint's tensor shapes")
        return int(self.shapes[name][0])

    @staticmethod
    def _mixed_attention(m: Dict) -> SeqLayer:
        s = SeqLayer()
        s.type = _lib.WF_SEQ_GQA_ATTENTION
        s.heads, s.dim, s.vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        s.kv_heads = int(m.get("kv_heads", s.heads))
        s.scale = float(m["scale"])
        s.window = int(m["mask"]["size"]) if m.get("mask") else NO_WINDOW
        s.qk_norm, s.proj_bias, s.head_gate, s.rope_dims = _lib.WF_SEQ_QKNORM_FULL, 0, 0, 0
        s.dist_log, s.sink, s.talk = 1, 2, 1
        return s

    def _gated_linear(self, m: Dict, prefix: str) -> SeqLayer:
        s = SeqLayer()
        s.type = _lib.WF_SEQ_GLA
        s.heads, s.dim, s.vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        s.decay_tau = float(m["tau"])
        s.decay_rank = self._rows(prefix + "a1", "the inner size of the decay projection")
        return s

    def native_layers(self) -> List[SeqLayer]:
        main, extra = [], []
        n = len(self.layers)
        for i, L in enumerate(self.layers):
            m, kind = L["mixer"], L["type"]
            if kind != "parallel":
                raise ValueError(f"config: layer {i} has unknown mixer type {kind!r}")
            s = self._mixed_attention(m["left"])
            s.pair = n + len(extra)
            s.pair_norm, s.mix_scale, s.pair_scale = 1, 0.5, 0.5
            extra.append(self._gated_linear(m["right"], f"l{i}.mix.right."))
            f = L.get("mlp")
            if f is None:
                s.has_ff = _lib.WF_SEQ_FF_NONE
            elif f.get("kind") == "dense":
                s.has_ff, s.ff_act, s.ff = _lib.WF_SEQ_FF_DENSE, _lib.WF_SEQ_ACT_GELU_TANH, int(f["ff"])
            else:
                raise ValueError(f"config: layer {i} has unknown feed-forward kind {f.get('kind')!r}")
            main.append(s)
        return main + extra


class FuvavikForCausalLM(SeqCausalLM):
    """Model class of the registry (weights, engine and step interface: wf_bitnet.seq_model.SeqCausalLM)."""

    architecture_names = ("Fuvavik", "FuvavikForCausalLM")
    reads_shapes = True

    @staticmethod
    def read_config(config: Dict, shapes: Optional[Dict[str, tuple]] = None) -> FuvavikConfig:
        return FuvavikConfig.from_dict(config, shapes)


EntryClass = FuvavikForCausalLM
