"""A plain, slow implementation of the Sisadra design in float64 torch on the CPU: the oracle of the tests.

One function per mechanism; whole sequences only (no cache, no state slots, no batches, no portions), so that
whatever the engine does with pages, slots and schedules is compared with something that has none of them.  It shares
no code with the product path.  `cfg` is the parsed config.json (a dict); `w` maps tensor names to float64 tensors.

Notation: n tokens, D = width; H query (or value) heads on G key/value (or query/key) heads, d = key size, e = value
size, R = latent size, T = taps of the short convolution.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch

F64 = torch.float64

# How much of a difference is rounding?  With `rounding_to(torch.bfloat16)` active, the values that a bfloat16 engine
# may keep in 16 bits (normalised rows, q, k, v, latents, the heads' outputs, activations) are rounded to that type on
# their way; the distance between such a run and the exact one is the noise that rounding alone causes, from which the
# tests take their bfloat16 tolerance.  Without it nothing is rounded.
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
def over_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return over_rms(x, eps) * weight


def centred_norm(x, weight, eps):
    """The mean is taken off; the variance is the mean of the squared deviations; no bias."""
    dev = x - x.mean(dim=-1, keepdim=True)
    return dev / torch.sqrt((dev * dev).mean(dim=-1, keepdim=True) + eps) * weight


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def capped(z, cap):
    return cap * torch.tanh(z / cap)


# ---- embedding ----------------------------------------------------------------------------------------------------
def pair_rows(tokens, bigram):
    """The row of the pair table for every token: a hash of the token before it and itself, the last row (behind the
    buckets) for the first."""
    rows = []
    for t, this in enumerate(tokens):
        rows.append(bigram["buckets"] if t == 0 else
                    (int(tokens[t - 1]) * bigram["mul_prev"] + int(this) * bigram["mul_cur"]) % bigram["buckets"])
    return torch.tensor(rows, dtype=torch.long)


def embed(tokens, w, cfg):
    emb = cfg["embedding"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * emb["scale"]
    if emb.get("bigram"):
        x = x + w["bigram"][pair_rows(list(tokens), emb["bigram"])]
    return x


# ---- rotation -----------------------------------------------------------------------------------------------------
def frequencies(rot):
    """[dims/2] frequencies base^(-2i/dims); where rot.scaling is given, waves longer than original/low are slowed down
    by `factor`, those shorter than original/high stay, and between the two the frequency is a mix of both."""
    dims, base = int(rot["dims"]), float(rot["base"])
    s = rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                keep = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - keep) * f / s["factor"] + keep * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x, positions, rot):
    """x [n, ..., d]: dimension i of the first rot.dims is turned together with dimension i + dims/2, the rest pass."""
    dims = int(rot["dims"])
    ang = torch.as_tensor(positions, dtype=F64)[:, None] * frequencies(rot)
    ang = ang.view(ang.shape[0], *([1] * (x.dim() - 2)), dims // 2)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * torch.cos(ang) - v * torch.sin(ang), v * torch.cos(ang) + u * torch.sin(ang), x[..., dims:]],
                     dim=-1)


# ---- differential attention within chunks ---------------------------------------------------------------------------
def same_chunk(n, size):
    """[n, n] bool: query i sees key j when j <= i and both lie in one chunk of `size` positions counted from 0 (None:
    every earlier key and itself)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i // size == j // size)


def masked_softmax(scores, seen):
    return torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)


def lambda_of(w, p, diff):
    return float(torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum())) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    """What the two maps of a head give, a1 and a2 [..., e], made one."""
    return over_rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, p, m, eps):
    """h [n, D] at positions 0 .. n-1; returns the mixer's output [n, D]."""
    n = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, 2, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, 2, d)
    v = kept(h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, e)
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    if m.get("rot"):
        q, k = rotate(q, range(n), m["rot"]), rotate(k, range(n), m["rot"])
    q, k = kept(q), kept(k)
    seen = same_chunk(n, m["mask"]["size"] if m.get("mask") else None)
    lam = lambda_of(w, p, m["diff"])
    heads = []
    for hh in range(H):
        g = hh // (H // G)
        a = [masked_softmax((q[:, hh, i] @ k[:, g, i].T) * m["scale"], seen) @ v[:, g] for i in (0, 1)]
        heads.append(difference_of_maps(a[0], a[1], lam, m["diff"], eps))
    return kept(torch.cat(heads, dim=-1)) @ w[p + "o"].T + w[p + "o.b"]


# ---- latent attention -----------------------------------------------------------------------------------------------
def sink_softmax(scores, seen, sink):
    """Softmax over the seen keys whose denominator also holds exp(sink): a slot without key and value."""
    s = scores.masked_fill(~seen, -math.inf)
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, torch.as_tensor(sink, dtype=F64))
    x = torch.exp(s - top)
    return x / (x.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, w, p, m, eps):
    n = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    c = kept(rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps))                 # [n, R]: all that is kept of a token
    q = (h @ w[p + "q"].T).view(n, H, d)
    k = (c @ w[p + "uk"].T).view(n, H, d)
    v = (c @ w[p + "uv"].T).view(n, H, e)
    seen = same_chunk(n, None)
    heads = [sink_softmax((q[:, i] @ k[:, i].T) * m["scale"], seen, w[p + "sink"][i]) @ v[:, i] for i in range(H)]
    return kept(torch.cat(heads, dim=-1)) @ w[p + "o"].T


# ---- the gated delta rule with a decay per key channel ----------------------------------------------------------------
def short_convolution(x, taps):
    """x [n, C], taps [C, T]: y[t, c] = sum_j taps[c, j] * x[t - (T-1) + j, c], zeros before the start."""
    n, T = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(T - 1, x.shape[1], dtype=x.dtype), x], dim=0)
    return sum(padded[j:j + n] * taps[:, j] for j in range(T))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def channel_decays(h, w, p, H, d):
    """[n, H, d]: exp(-exp(A_log) softplus(W2 W1 h + dt_bias)), one per head and key channel."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z).view(-1, H, d))


def delta_rule(q, k, v, beta, decay):
    """One head: q, k, decay [n, d], v [n, e], beta [n].  The state S [d, e] starts at zero; for each token its rows decay,
    then u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.T @ q[t])
    return torch.stack(out)


def channel_delta(h, w, p, m, eps):
    n = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_convolution(h @ w[p + "q"].T, w[p + "q.conv"])).view(n, G, d)
    k = silu(short_convolution(h @ w[p + "k"].T, w[p + "k.conv"])).view(n, G, d)
    v = silu(short_convolution(h @ w[p + "v"].T, w[p + "v.conv"])).view(n, H, e)
    q, k = unit_vector(q) * d ** -0.5, unit_vector(k)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    decay = channel_decays(h, w, p, H, d)
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(n, H, e)
    heads = []
    for hh in range(H):
        g = hh // (H // G)
        o = delta_rule(q[:, g], k[:, g], v[:, hh], beta[:, hh], decay[:, hh])
        heads.append(rms_norm(o, w[p + "norm"], eps) * gate[:, hh])
    return kept(torch.cat(heads, dim=-1)) @ w[p + "o"].T


MIXERS = {"attention": differential_attention, "latent_attention": latent_attention, "channel_delta": channel_delta}


# ---- the model ---------------------------------------------------------------------------------------------------
def dense(h, w, p):
    return kept(gelu(h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, w, tokens, layer_outputs=None):
    """Logits [n, vocab] of one whole sequence; `layer_outputs` (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w, cfg)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[L["type"]](kept(centred_norm(x, w[p + "norm1"], eps)), w, p + "mix.", L["mixer"], eps)
        if L.get("mlp") is not None:
            x = x + dense(kept(centred_norm(x, w[p + "norm2"], eps)), w, p + "mlp.")
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    logits = kept(centred_norm(x, w["final.norm"], eps)) @ w["head"].T
    return capped(logits, cfg["logit_softcap"]) if cfg.get("logit_softcap") else logits


def rounding_noise(cfg, w, tokens, dtype=torch.bfloat16):
    """Per position, the largest difference between the logits with the 16-bit values rounded and the exact ones, as a
    fraction of the largest exact logit: (the largest over the positions, their median)."""
    exact = forward(cfg, w, tokens)
    with rounding_to(dtype):
        rounded = forward(cfg, w, tokens)
    per_row = (rounded - exact).abs().max(dim=1).values / exact.abs().max()
    return float(per_row.max()), float(per_row.median())


# ---- a safetensors reader of its own -----------------------------------------------------------------------------------
def read_safetensors(path) -> dict:
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    out = {}
    for name, meta in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        buf = raw[8 + n + lo:8 + n + hi]
        if meta["dtype"] == "BF16":
            a = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif meta["dtype"] == "F32":
            a = np.frombuffer(buf, dtype="<f4").astype(np.float64)
        else:
            raise ValueError(f"{name}: dtype {meta['dtype']}")
        out[name] = torch.from_numpy(a.reshape(meta["shape"]).copy())
    return out


def read_folder(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")
