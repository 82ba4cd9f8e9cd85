"""A plain, slow implementation of the Saropel design in float64 torch on the CPU: the oracle of the tests.

One function per mechanism; whole sequences only (no cache, no pages, no batches, no portions), so that whatever the
engine does with pages and schedules is compared with something that has none of them.  It shares no code with the
product path.  `cfg` is the parsed config.json (a dict); `w` maps tensor names to float64 tensors.

Notation: n tokens, D = width.  Attention: H query heads on G key/value heads, d = query/key size, e = value size,
R = rotated dimensions of a head, W = window.  Feed-forward: E experts in C groups, K experts a token.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch

F64 = torch.float64

# With `rounding_to(torch.bfloat16)` active, the values that a bfloat16 engine may keep in 16 bits (the inputs of
# products, cached rows, activations) are rounded to that type on their way; the distance between such a run and the
# exact one is the noise that rounding alone causes, from which the tests take their bfloat16 tolerance.
_ROUND = [None]


class rounding_to:
    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        _ROUND[0] = self.dtype

    def __exit__(self, *exc):
        _ROUND[0] = None


def kept(x):
    return x if _ROUND[0] is None else x.to(_ROUND[0]).to(F64)


# ---- small mechanisms -------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x, weight, eps):
    """The stored weight is the deviation from one."""
    return unit_rms(x, eps) * (1.0 + weight)


def norm_plain(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- embedding ----------------------------------------------------------------------------------------------------
def pair_rows(tokens, bigram):
    """The row of the pair table for every token: a hash of the token before it and itself, the last row (behind the
    buckets) for the first."""
    rows = [bigram["buckets"]]
    for before, this in zip(tokens[:-1], tokens[1:]):
        rows.append((int(before) * bigram["mul_prev"] + int(this) * bigram["mul_cur"]) % bigram["buckets"])
    return torch.tensor(rows[:len(tokens)], dtype=torch.long)


def embed(tokens, w, cfg):
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        x = x + w["bigram"][pair_rows(list(tokens), bigram)]
    return x


# ---- rotation -----------------------------------------------------------------------------------------------------
def frequencies(rot):
    """([dims/2] frequencies, factor on cos and sin): base^(-2i/dims), the slow ones stretched where rot.scaling says
    so."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=F64), 1.0

    def pair_with_turns(t):
        return dims * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_with_turns(s["fast"])), 0)
    hi = min(math.ceil(pair_with_turns(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [n, heads, d]: dimension i of the first rot.dims is turned together with dimension i + dims/2, the rest pass."""
    dims = int(rot["dims"])
    f, magnitude = frequencies(rot)
    ang = torch.as_tensor(positions, dtype=F64)[:, None, None] * f
    cos, sin = magnitude * torch.cos(ang), magnitude * torch.sin(ang)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


# ---- attention ----------------------------------------------------------------------------------------------------
def visible(n, window):
    """[n, n] bool: query i sees key j when 0 <= i - j < window (None: every earlier key and itself)."""
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    seen = back >= 0
    return seen if window is None else seen & (back < window)


def capped(scores, cap):
    return scores if cap is None else cap * torch.tanh(scores / cap)


def attend(q, k, v, scale, window, cap=None):
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e]."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    group = torch.arange(H) // (H // G)
    scores = capped(torch.einsum("ihd,jhd->hij", q, k[:, group]) * scale, cap)
    a = torch.softmax(scores.masked_fill(~visible(n, window)[None], -math.inf), dim=-1)
    return torch.einsum("hij,jhe->ihe", a, v[:, group])


def window_of(m):
    return m["mask"]["size"] if m.get("mask") else None


def capped_attention(h, w, p, m):
    """No rotation; scores pass a soft cap."""
    n, hk = h.shape[0], kept(h)
    q = kept((hk @ w[p + "q"].T).reshape(n, m["heads"], m["dim"]))
    k = kept((hk @ w[p + "k"].T).reshape(n, m["kv_heads"], m["dim"]))
    v = kept((hk @ w[p + "v"].T).reshape(n, m["kv_heads"], m["vdim"]))
    o = attend(q, k, v, m["scale"], window_of(m), m.get("softcap"))
    return kept(o).reshape(n, -1) @ w[p + "o"].T


def shared_kv_attention(h, w, p, m, eps, positions):
    """The values are the projected keys; queries and keys pass a norm per head and a rotation; one gate per head."""
    n, hk = h.shape[0], kept(h)
    q = (hk @ w[p + "q"].T).reshape(n, m["heads"], m["dim"])
    k = (hk @ w[p + "k"].T).reshape(n, m["kv_heads"], m["dim"])
    v = kept(k)
    q = norm_plain(q, w[p + "q.norm"], eps)
    k = norm_plain(k, w[p + "k.norm"], eps)
    if m.get("rot") and m["rot"].get("dims"):
        q, k = rotate(q, positions, m["rot"]), rotate(k, positions, m["rot"])
    o = attend(kept(q), kept(k), v, m["scale"], window_of(m))
    o = kept(o) * torch.sigmoid(hk @ w[p + "g"].T)[:, :, None]
    return kept(o).reshape(n, -1) @ w[p + "o"].T


# ---- feed-forwards ------------------------------------------------------------------------------------------------
def dense_ff(h, w, p):
    hk = kept(h)
    return kept(silu(hk @ w[p + "gate"].T) * (hk @ w[p + "up"].T)) @ w[p + "down"].T


def limited_expert(h, w, p, limit):
    hk = kept(h)
    g = torch.clamp(hk @ w[p + "gate"].T, max=limit)
    u = torch.clamp(hk @ w[p + "up"].T, -limit, limit)
    return kept(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(scores, router):
    """(chosen [n, K], weights [n, K]) from scores [n, E]: only experts of the best groups.keep groups (a group's score
    is its largest) may be chosen; the K largest of them, the lower index on a tie, weigh as they are."""
    n, E = scores.shape
    allowed = scores.clone()
    groups = router.get("groups")
    if groups:
        per = E // groups["count"]
        best = scores.reshape(n, groups["count"], per).max(dim=-1).values
        kept_groups = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, :groups["keep"]]
        mask = torch.zeros(n, groups["count"], dtype=torch.bool).scatter_(1, kept_groups, True)
        allowed = scores.masked_fill(~mask.repeat_interleave(per, dim=1), -1.0)
    order = torch.sort(allowed, dim=-1, descending=True, stable=True).indices[:, :router["top"]]
    return order, torch.gather(scores, 1, order)


def routed_ff(h, w, p, mlp):
    scores = torch.softmax(kept(h) @ w[p + "router"].T, dim=-1)
    chosen, weights = choose(scores, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(chosen.shape[1]):
            e = int(chosen[t, j])
            out[t] += weights[t, j] * limited_expert(h[t:t + 1], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        gate = torch.sigmoid(kept(h) @ w[p + "shared.sg"].T)
        out = out + gate * limited_expert(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


def feed_forward(h, w, p, mlp):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else routed_ff(h, w, p, mlp)


# ---- what a token gives to every layer ------------------------------------------------------------------------------
def token_input(x, tokens, i, w, p, dim, eps):
    """x + norm(proj(gelu(gate x) * e)), e the layer's part of the token's row."""
    e = w["side.embed"][torch.as_tensor(tokens, dtype=torch.long), i * dim:(i + 1) * dim]
    g = kept(gelu_tanh(kept(x) @ w[p + "side.gate"].T) * e)
    return x + norm_plain(g @ w[p + "side.proj"].T, w[p + "side.norm"], eps)


# ---- the model ------------------------------------------------------------------------------------------------------
def run_order(cfg):
    """(layer, pass that begins right before it or None) in the order of the run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def layer(x, tokens, i, cfg, w):
    L, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    h = norm_around_one(x, w[p + "norm1"], eps)
    if L["type"] == "attention":
        y = capped_attention(h, w, p + "mix.", L["mixer"])
    elif L["type"] == "attention_2":
        y = shared_kv_attention(h, w, p + "mix.", L["mixer"], eps, range(len(tokens)))
    else:
        raise ValueError(f"unknown mixer {L['type']!r}")
    if L.get("mlp") is not None:
        y = y + feed_forward(h, w, p + "mlp.", L["mlp"])
    x = x + y
    if cfg.get("token_side"):
        x = token_input(x, tokens, i, w, p, cfg["token_side"]["dim"], eps)
    return x


def forward(cfg: dict, w: dict, tokens, collect=None):
    """Logits [n, vocab] of one whole sequence.  `collect` (a list) receives the stream after every layer run."""
    x0 = embed(tokens, w, cfg)
    x = x0
    for i, begins in run_order(cfg):
        if begins is not None:
            if begins > 0:
                x = x + x0
            x = x + w["loop.step"][begins]
        x = layer(x, tokens, i, cfg, w)
        if collect is not None:
            collect.append(x.clone())
    return kept(norm_around_one(x, w["final.norm"], cfg["norm"]["eps"])) @ w["head"].T


def rounding_noise(cfg, w, tokens, dtype=torch.bfloat16):
    """Per position, the largest difference between the logits with the 16-bit values rounded and the exact ones, as a
    fraction of the largest exact logit: (the largest over the positions, their median)."""
    exact = forward(cfg, w, tokens)
    with rounding_to(dtype):
        rounded = forward(cfg, w, tokens)
    per_row = (rounded - exact).abs().max(dim=1).values / exact.abs().max()
    return float(per_row.max()), float(per_row.median())


# ---- reading a model folder -----------------------------------------------------------------------------------------
def read_folder(folder):
    """(cfg, w): config.json as a dict and every tensor of model.safetensors as float64 (own parser)."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    (hlen,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + hlen])
    w = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        buf = raw[8 + hlen + lo:8 + hlen + hi]
        if info["dtype"] == "BF16":
            u = np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(u.view(np.float32).astype(np.float64))
        elif info["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(buf, dtype="<f4").astype(np.float64))
        elif info["dtype"] == "I32":
            t = torch.from_numpy(np.frombuffer(buf, dtype="<i4").astype(np.int64))
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
        w[name] = t.reshape(info["shape"])
    return cfg, w
