"""Plain, slow statement of the Kilizen design in PyTorch (float64), one function per mechanism, whole sequences at once with the
recurrence as a Python loop over the tokens.  It shares no code with the serving path: the GPU tests compare the engine with these
functions.

A model is a config dict (the shape of config.json) and a dict of tensors by checkpoint name.  Every sublayer sits between two
element-wise norms tanh(alpha x) w + b: x <- x + n1b(mixer(n1(x))), x <- x + n2b(ff(n2(x))).  A range of layers can run several times in a
row with the same weights; before each pass but the first the embedding is added to the stream.  Mixers:
  'attention'    grouped-query attention whose values are its keys as projected, RMS norm per query / key head, a partial half-split
                 rotation with frequency interpolation, a sliding window beside a few first positions that stay visible, learned sinks;
  'attention_2'  causal grouped-query attention with biased projections, RMS norm over the whole query / key projection, a half-split
                 rotation, learned sinks;
  'mlstm'        matrix memory with exponential input gate, sigmoid forget gate and a running maximum of the log gates.
The feed-forward is down(gelu(up h)), or routed experts down(relu(up h)^2) weighted by a softmax over the chosen logits plus a shared expert.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

DT = torch.float64


def dyn_tanh(x: torch.Tensor, w: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    """The norm without statistics."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_exact(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.special.erf(z / math.sqrt(2.0)))


def relu_sq(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


# ---- rotation
def turn_rates(rot: Dict) -> Tuple[torch.Tensor, float]:
    """Angle per position of every rotated pair, and the factor on cosines and sines."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=DT)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    edge = lambda turns: dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(edge(float(sc["fast"]))), 0)
    hi = min(math.ceil(edge(float(sc["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    factor = float(sc["factor"])
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_half(x: torch.Tensor, pos: torch.Tensor, rot: Optional[Dict]) -> torch.Tensor:
    """x [T, heads, d]: entries i and i + dims / 2 turned together, the rest unchanged."""
    if not rot or not int(rot["dims"]):
        return x
    f, mag = turn_rates(rot)
    half = int(rot["dims"]) // 2
    a = pos.to(DT)[:, None] * f[None, :]
    c, s = (torch.cos(a) * mag)[:, None, :], (torch.sin(a) * mag)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ---- attention
def visible(T: int, mask: Optional[Dict]) -> torch.Tensor:
    """[T, T] bool: does position i see position j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask:
        seen = seen & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return seen


def sink_softmax(s: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Softmax over the last axis whose denominator also holds exp(sink)."""
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, seen: torch.Tensor, scale: float, sink: torch.Tensor) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        s = torch.where(seen, s, torch.full_like(s, -math.inf))
        out.append(sink_softmax(s, sink[h]) @ v[:, h // rep])
    return torch.stack(out, 1).reshape(T, -1)


def window_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    raw = (h @ w[p + "k"].T).view(T, G, d)                        # the values: keys before norm and rotation
    q = unit_rms((h @ w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"]
    k = unit_rms(raw, eps) * w[p + "k.norm"]
    q, k = rotate_half(q, pos, m.get("rot")), rotate_half(k, pos, m.get("rot"))
    return attend(q, k, raw, visible(T, m.get("mask")), m["scale"], w[p + "sink"]) @ w[p + "o"].T


def full_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = unit_rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]          # one norm over all heads
    k = unit_rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    q, k = rotate_half(q.view(T, H, d), pos, m.get("rot")), rotate_half(k.view(T, G, d), pos, m.get("rot"))
    return attend(q, k, v, visible(T, m.get("mask")), m["scale"], w[p + "sink"]) @ w[p + "o"].T + w[p + "o.b"]


# ---- matrix memory
def log_logistic(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def matrix_memory(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q = (h @ w[p + "q"].T).view(T, H, d) / math.sqrt(d)
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    gi = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    gf = log_logistic(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    S, n, top = torch.zeros(H, d, dv, dtype=DT), torch.zeros(H, d, dtype=DT), torch.zeros(H, dtype=DT)
    rows = []
    for t in range(T):
        new = torch.maximum(gf[t] + top, gi[t])
        keep, put = torch.exp(gf[t] + top - new), torch.exp(gi[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        top = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        rows.append((S * q[t][:, :, None]).sum(1) / den[:, None])
    o = unit_rms(torch.stack(rows), eps).reshape(T, H * dv)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward
def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return gelu_exact(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return relu_sq(h @ w[p + "up"].T) @ w[p + "down"].T


def choose(z: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Logits [T, N] -> (expert indices [T, top], weights [T, top]): softmax over the chosen logits alone."""
    val, idx = z.topk(top, dim=-1)
    e = torch.exp(val - val[:, :1])
    return idx, e / e.sum(-1, keepdim=True)


def routed_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, f: Dict) -> torch.Tensor:
    idx, wt = choose(h @ w[p + "router"].T, f["router"]["top"])
    y = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if t.numel():
            y[t] += wt[t, k][:, None] * expert(h[t], w, f"{p}e{e}.")
    return y + expert(h, w, p + "shared.") if f.get("shared") else y


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, f: Dict) -> torch.Tensor:
    return dense_ff(h, w, p) if f["kind"] == "dense" else routed_ff(h, w, p, f)


# ---- layer, model
MIXERS = {"attention": window_attention, "attention_2": full_attention, "mlstm": matrix_memory}


def layer(x: torch.Tensor, w: Dict[str, torch.Tensor], i: int, L: Dict, eps: float) -> torch.Tensor:
    p = f"l{i}."
    x = x + dyn_tanh(MIXERS[L["type"]](dyn_tanh(x, w, p + "norm1"), w, p + "mix.", L["mixer"], eps), w, p + "norm1b")
    if L.get("mlp"):
        x = x + dyn_tanh(feed_forward(dyn_tanh(x, w, p + "norm2"), w, p + "mlp.", L["mlp"]), w, p + "norm2b")
    return x


def layer_runs(cfg: Dict) -> List[Tuple[int, bool]]:
    """The layers in the order they run: (layer, is the embedding added right before it)."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(lp["times"]):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg: Dict, w: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """-> logits [T, vocab]; taps (optional list) receives the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    emb = w["embed"][torch.tensor(tokens)]
    x = emb
    for i, again in layer_runs(cfg):
        if again:
            x = x + emb
        x = layer(x, w, i, cfg["layers"][i], eps)
        if taps is not None:
            taps.append(x.clone())
    return dyn_tanh(x, w, "final.norm") @ w["head"].T


def random_weights(cfg: Dict, seed: int = 0, sharp: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random tensors with the checkpoint's names and shapes, values representable in bfloat16.  `sharp` scales the weights of the
    queries' norm (sharper softmax)."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out: Dict[str, torch.Tensor] = {}

    def mat(name, o, i, s=None):
        out[name] = (torch.randn(o, i, generator=g) * (s if s is not None else 1.0 / math.sqrt(i))).bfloat16().float()

    def vec(name, n, s=0.1, mean=0.0):
        out[name] = (mean + torch.randn(n, generator=g) * s).bfloat16().float()

    def norm(name, lo=0.4, hi=1.2):
        vec(name, W, 0.2, 1.0)
        vec(name + ".b", W, 0.1)
        out[name + ".alpha"] = (lo + (hi - lo) * torch.rand((), generator=g)).bfloat16().float()

    out["embed"] = torch.randn(V, W, generator=g).bfloat16().float()
    norm("final.norm")
    mat("head", V, W)
    for li, L in enumerate(cfg["layers"]):
        p, m, q = f"l{li}.", L["mixer"], f"l{li}.mix."
        norm(p + "norm1")
        norm(p + "norm1b")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "mlstm":
            mat(q + "q", H * d, W); mat(q + "k", H * d, W); mat(q + "v", H * dv, W); mat(q + "g", H * dv, W)
            mat(q + "i", H, W, 1.5 / math.sqrt(W)); vec(q + "i.b", H, 0.5)
            mat(q + "f", H, W, 1.5 / math.sqrt(W)); vec(q + "f.b", H, 0.5, 2.0)
            vec(q + "norm", H * dv, 0.1, 1.0)
        else:
            G = m["kv_heads"]
            two = L["type"] == "attention_2"
            mat(q + "q", H * d, W); mat(q + "k", G * d, W)
            vec(q + "q.norm", H * d if two else d, 0.1, sharp); vec(q + "k.norm", G * d if two else d, 0.1, 1.0)
            vec(q + "sink", H, 1.0)
            if two:
                mat(q + "v", G * dv, W)
                vec(q + "q.b", H * d, 0.3); vec(q + "k.b", G * d, 0.3); vec(q + "v.b", G * dv, 0.3); vec(q + "o.b", W, 0.3)
        mat(q + "o", W, H * dv)
        f = L.get("mlp")
        if f is None:
            continue
        norm(p + "norm2")
        norm(p + "norm2b")
        r = p + "mlp."
        if f["kind"] == "dense":
            mat(r + "up", f["ff"], W); mat(r + "down", W, f["ff"])
            continue
        mat(r + "router", f["router"]["experts"], W, 2.0 / math.sqrt(W))
        names = [(f"e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        for n, ff in names + ([("shared.", f["shared"]["ff"])] if f.get("shared") else []):
            mat(r + n + "up", ff, W); mat(r + n + "down", W, ff)
    return out
