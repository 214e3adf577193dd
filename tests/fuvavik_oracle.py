"""Plain, slow statement of the Fuvavik design in PyTorch (float64), one function per mechanism, whole sequences at once with the
recurrence as a Python loop over the tokens.  It shares no code with the serving path: the GPU tests compare the engine with these
functions.

A model is a config dict (the shape of config.json) and a dict of tensors by checkpoint name.  The stream starts as the scaled embedding
plus a learned vector per position.  A layer has ONE layer norm (mean taken off, weight and bias) whose output h both branches read; each
branch's result is multiplied element by element by a gate computed from h:  x <- x + s(R1 h + b1) * mixer(h) + s(R2 h + b2) * ff(h).
The mixer is a pair on the same input, half the sum of both after an RMS norm of each:
  left   grouped-query sliding-window attention: query / key norm over the whole projection, no rotation, a logarithmic distance penalty,
         a learned sink per head, and the heads' softmax weights mixed by a matrix before they meet the values;
  right  gated linear attention: a matrix state per head whose key rows decay each by its own factor.
The feed-forward is down(gelu_tanh(gate h) * (up h)); the head is the embedding table, its logits capped by a tanh.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensors = Dict[str, torch.Tensor]


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x * (x.pow(2).mean(-1, keepdim=True) + eps).rsqrt()


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(-1, keepdim=True)
    return c * (c.pow(2).mean(-1, keepdim=True) + eps).rsqrt() * w + b


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return z * 0.5 * (torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z.pow(3))) + 1.0)


def embed(tokens: List[int], w: Tensors, scale: float, pos0: int = 0) -> torch.Tensor:
    return w["embed"][torch.tensor(tokens)] * scale + w["pos"][pos0:pos0 + len(tokens)]


# ---- left: window attention with mixed heads
def log_penalty(dist: torch.Tensor, r1: torch.Tensor, r2: torch.Tensor) -> torch.Tensor:
    """What is taken off a score at a distance: r1 ln(1 + r2 distance)."""
    return r1 * torch.log1p(r2 * dist)


def softmax_with_sink(s: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Weights over the last axis; the sink takes its share of the sum and appears nowhere else."""
    top = torch.maximum(s.amax(-1, keepdim=True), sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def head_weights(h: torch.Tensor, w: Tensors, p: str, m: Dict, eps: float) -> torch.Tensor:
    """The heads' softmax weights before they are mixed, [H, T, T]."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(h.dtype)
    span = m["mask"]["size"] if m.get("mask") else T
    hidden = (dist < 0) | (dist >= span)
    out = []
    for hd in range(H):
        s = (q[:, hd] @ k[:, hd * G // H].T) * m["scale"] - log_penalty(dist.clamp(min=0), w[p + "r1"][hd], w[p + "r2"][hd])
        out.append(softmax_with_sink(s.masked_fill(hidden, -math.inf), w[p + "sink"][hd]))
    return torch.stack(out)


def mixed_attention(h: torch.Tensor, w: Tensors, p: str, m: Dict, eps: float) -> torch.Tensor:
    T, H, G, dv = h.shape[0], m["heads"], m["kv_heads"], m["vdim"]
    v = (h @ w[p + "v"].T).view(T, G, dv)
    a = torch.einsum("hg,gij->hij", w[p + "talk"], head_weights(h, w, p, m, eps))
    o = torch.stack([a[hd] @ v[:, hd * G // H] for hd in range(H)], 1)
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---- right: gated linear attention
def channel_decay(h: torch.Tensor, w: Tensors, p: str, tau: float) -> torch.Tensor:
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gated_linear(h: torch.Tensor, w: Tensors, p: str, m: Dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) / math.sqrt(d)
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    a = channel_decay(h, w, p, m["tau"]).view(T, H, d)
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    rows = []
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hkv,hk->hv", S, q[t]))
    o = unit_rms(torch.stack(rows), eps) * w[p + "norm"]
    return (o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def pair(h: torch.Tensor, w: Tensors, p: str, m: Dict, eps: float) -> torch.Tensor:
    a = unit_rms(mixed_attention(h, w, p + "left.", m["left"], eps), eps) * w[p + "left.out"]
    b = unit_rms(gated_linear(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return (a + b) / 2


# ---- feed-forward, layer, model
def dense_ff(h: torch.Tensor, w: Tensors, p: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def branch_gate(h: torch.Tensor, w: Tensors, name: str) -> torch.Tensor:
    return torch.sigmoid(h @ w[name].T + w[name + ".b"])


def layer(x: torch.Tensor, w: Tensors, i: int, L: Dict, eps: float) -> torch.Tensor:
    p = f"l{i}."
    h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
    y = branch_gate(h, w, p + "rg1") * pair(h, w, p + "mix.", L["mixer"], eps)
    if L.get("mlp"):
        y = y + branch_gate(h, w, p + "rg2") * dense_ff(h, w, p + "mlp.")
    return x + y


def forward(cfg: Dict, w: Tensors, tokens: List[int], taps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """-> logits [T, vocab]; taps (optional list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = embed(tokens, w, float(cfg["embedding"]["scale"]))
    for i, L in enumerate(cfg["layers"]):
        x = layer(x, w, i, L, eps)
        if taps is not None:
            taps.append(x.clone())
    lg = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(lg / cap) if cap else lg


def random_weights(cfg: Dict, seed: int = 0, ranks: Optional[Dict[int, int]] = None) -> Tensors:
    """Random tensors with the checkpoint's names and shapes, values representable in bfloat16.  ranks[layer]: the inner size of the
    two-matrix decay projection (config.json leaves it to the tensors' shapes)."""
    gen = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out: Tensors = {}

    def put(name, shape, spread, mean=0.0):
        out[name] = (mean + torch.randn(*shape, generator=gen) * spread).bfloat16().float()

    def mat(name, o, i):
        put(name, (o, i), i ** -0.5)

    put("embed", (V, W), 0.5)
    put("pos", (cfg["max_positions"], W), 0.3)
    put("final.norm", (W,), 0.2, 1.0)
    put("final.norm.b", (W,), 0.2)
    for li, L in enumerate(cfg["layers"]):
        p, a, r = f"l{li}.", L["mixer"]["left"], L["mixer"]["right"]
        put(p + "norm1", (W,), 0.2, 1.0)
        put(p + "norm1.b", (W,), 0.2)
        q = p + "mix.left."
        H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        mat(q + "q", H * d, W); mat(q + "k", G * d, W); mat(q + "v", G * dv, W); mat(q + "o", W, H * dv)
        put(q + "q.norm", (H * d,), 0.2, 1.0); put(q + "k.norm", (G * d,), 0.2, 1.0)
        out[q + "r1"] = (0.2 + 0.8 * torch.rand(H, generator=gen)).bfloat16().float()
        out[q + "r2"] = (0.1 + 1.5 * torch.rand(H, generator=gen)).bfloat16().float()
        put(q + "sink", (H,), 0.7)
        out[q + "talk"] = (torch.eye(H) * 0.8 + torch.randn(H, H, generator=gen) * 0.4).bfloat16().float()
        q = p + "mix.right."
        H, d, dv, k = r["heads"], r["dim"], r["vdim"], (ranks or {}).get(li, 8)
        mat(q + "q", H * d, W); mat(q + "k", H * d, W); mat(q + "v", H * dv, W); mat(q + "g", H * dv, W); mat(q + "o", W, H * dv)
        put(q + "norm", (dv,), 0.1, 1.0)
        mat(q + "a1", k, W); mat(q + "a2", H * d, k); put(q + "a2.b", (H * d,), 1.0, 1.0)
        put(p + "mix.left.out", (W,), 0.2, 1.0); put(p + "mix.right.out", (W,), 0.2, 1.0)
        mat(p + "rg1", W, W); put(p + "rg1.b", (W,), 0.5)
        if L.get("mlp"):
            f = L["mlp"]["ff"]
            mat(p + "mlp.gate", f, W); mat(p + "mlp.up", f, W); mat(p + "mlp.down", W, f)
            mat(p + "rg2", W, W); put(p + "rg2.b", (W,), 0.5)
    return out
