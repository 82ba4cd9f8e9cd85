"""Sisadra on the GPU against the plain implementation (tests/plain_sisadra.py): each mechanism alone through its kernels
and parts, then whole models under schedules (whole, token by token, portions down to two tokens, mixed batches on a pool
so small that pages and slots are used again), the edges of chunks in prompts and in decoding, states and the token before
across steps and slots, a far key among hundreds, long decoding, random configurations, and greedy generation through
generate()."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_sisadra as ps
import sisadra_tiny as st
import tiny
from test_fegizen_gpu import fake_batch
from test_tubepel_gpu import STEPS, compare, i32, rel_err, run_mixer_in_steps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


# ---------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [8, 50, 256, 4100])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_centring_norm_with_a_bias_that_joins_the_stream(width, dtype):
    """The bias with shares, with nothing pending (a product that has added to the stream itself), and over chosen rows,
    where nothing is written back."""
    from flambeau_b200.kernels import ops
    n, eps = 11, 1e-3
    g = torch.Generator().manual_seed(width)
    dt = DT[dtype]
    x, d = torch.randn(n, width, generator=g) + 3.0, torch.randn(3, n, width, generator=g)
    w, b = (torch.randn(width, generator=g).to(dt) for _ in range(2))
    rows = [7, 0, 3]
    for delta, bias, chosen in ((d, b, None), (None, b, None), (d, None, None), (d, b, rows), (None, b, rows), (None, None, None)):
        xd, out = x.to(DEV), torch.empty(len(chosen) if chosen else n, width, dtype=dt, device=DEV)
        dd = delta.to(DEV) if delta is not None else None
        ops.add_layer_norm(xd, dd[0] if dd is not None else None, w.to(DEV), eps, out, rows=i32(chosen) if chosen else None,
                           n_partials=3 if dd is not None else 1, partial_stride=dd.stride(0) if dd is not None else 0,
                           delta_bias=bias.to(DEV) if bias is not None else None)
        v = x.double() + (delta.double().sum(0) if delta is not None else 0) + (bias.double() if bias is not None else 0)
        want = ps.centred_norm(v[chosen] if chosen else v, w.double(), eps)
        assert rel_err(out, want) < (5e-6 if dtype == "float32" else 6e-3)
        assert rel_err(xd, x.double() if chosen else v) < 1e-6, "written back exactly where all rows are formed"


@pytest.mark.parametrize("shape", [(1, 7), (5, 40), (300, 1000)], ids=str)
def test_exact_gelu_and_capped_logits(shape):
    from flambeau_b200.kernels import ops
    n, cols = shape
    g = torch.Generator().manual_seed(n)
    z = torch.randn(3, n, cols, generator=g) * 2.0
    zd = z.to(DEV)
    for dtype in DT.values():
        out = torch.empty(n, cols, dtype=dtype, device=DEV)
        ops.activation(zd[0], out, "gelu", n_partials=3, partial_stride=zd.stride(0))
        assert rel_err(out, ps.gelu(z.double().sum(0))) < (1e-6 if dtype == torch.float32 else 4e-3)
    x = torch.linspace(-90.0, 90.0, n * cols).view(n, cols)
    wide = torch.full((n, cols + 3), 7.0)
    wide[:, :cols] = x
    wd = wide.to(DEV)
    ops.softcap_rows(wd[:, :cols], 30.0)
    assert rel_err(wd[:, :cols], ps.capped(x.double(), 30.0)) < 1e-6 and bool((wd[:, cols:] == 7.0).all())


@pytest.mark.parametrize("shape", [(5, 64, 40), (64, 96, 40), (130, 64, 80), (600, 256, 512)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_plain_feed_forward_with_the_exact_gelu(shape, dtype):
    """Few rows (shares and the activation kernel) and many (the activation in the product's epilogue)."""
    from test_parts_gpu import Bench, bind_random
    from flambeau_b200.parts.feedforward import PlainMLP
    n, D, ff = shape
    b = Bench(dtype, max_step_tokens=1024, cache_tokens=1024)
    part = PlainMLP(b.rt, "m.", width=D, inner=ff, activation="gelu", init_std=0.2)
    Wt = bind_random(part, DT[dtype])
    h = torch.randn(n, D, generator=torch.Generator().manual_seed(n)).to(DT[dtype])
    ctx, _ = b.begin([("a", [1] * n, [])], D)
    ctx.pending_slabs = 1
    part.forward(ctx, h.to(DEV), ctx.delta)
    b.end()
    out = ctx.delta_slabs[:ctx.pending_slabs].sum(0)
    assert rel_err(out, ps.dense(h.double(), Wt, "m.")) < (2e-5 if dtype == "float32" else 2e-2)


# (heads, kv heads, key size per map, value size, rotated dimensions)
MAP_SIZES = [(4, 2, 32, 48, 8), (3, 1, 16, 8, 16), (6, 3, 48, 96, 20), (5, 5, 10, 18, 6), (2, 1, 64, 64, 32), (2, 2, 160, 96, 40),
             (1, 1, 6, 10, 0), (18, 1, 16, 32, 12), (1, 1, 128, 256, 128)]


@pytest.mark.parametrize("sizes", MAP_SIZES, ids=str)
@pytest.mark.parametrize("n", [9, 90])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_maps_are_biased_normed_turned_and_written_side_by_side(sizes, n, dtype):
    """Projection rows as shares -> q, and the cache's key rows with both maps of a head side by side.  Biases that move
    the norms; weights of the norms far from one; with and without norm and bias."""
    from flambeau_b200.cache.manager import LayerCacheView
    from flambeau_b200.kernels import ops
    H, G, d, e, rot = sizes
    dt, page, eps, base = DT[dtype], 8, 1e-3, 300.0
    g = torch.Generator().manual_seed(d)
    positions = [int(p) for p in torch.randperm(40 * page, generator=g)[:n]]
    cols = (H + G) * 2 * d + G * e
    pad = -(-cols // 8) * 8
    shares = torch.randn(3, n, pad, generator=g)
    bias = (torch.randn(cols, generator=g) * 2.0).to(dt)
    qw, kw = ((torch.randn(d, generator=g) + 2.0).to(dt) for _ in range(2))
    table = torch.randperm(40, generator=g).to(torch.int32)
    freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64)
    ang = torch.tensor(positions, dtype=F64)[:, None] * freq[None] if rot else None
    tables = (torch.cos(ang).float().to(DEV), torch.sin(ang).float().to(DEV)) if rot else (None, None)
    sh = shares.to(DEV)
    for with_norm, with_bias in ((True, True), (True, False), (False, True)):
        x = shares.double().sum(0)[:, :cols] + (bias.double() if with_bias else 0)
        q, k = x[:, :2 * H * d].view(n, H, 2, d), x[:, 2 * H * d:2 * (H + G) * d].view(n, G, 2, d)
        v = x[:, 2 * (H + G) * d:].view(n, G, e)
        if with_norm:
            q, k = ps.rms_norm(q, qw.double(), eps), ps.rms_norm(k, kw.double(), eps)
        if rot:
            q, k = (ps.rotate(t, positions, {"dims": rot, "base": base}) for t in (q, k))
        cache = LayerCacheView(torch.zeros((40, G, page, 2 * d), dtype=dt, device=DEV), torch.zeros((40, G, page, e), dtype=dt, device=DEV),
                               table[None].to(DEV).contiguous(), i32([0]), page, True, 0, None)
        q_out, status = torch.empty((n, 2 * H * d), dtype=dt, device=DEV), i32([0])
        ops.qk_norm_rope_kv_write(sh[0], qw.to(DEV) if with_norm else None, kw.to(DEV) if with_norm else None,
                                  "head" if with_norm else None, eps, 0.0, *tables, rot // 2, q_out, cache, i32(positions),
                                  i32([0] * n), 2 * H, 2 * G, d, e, status, n_partials=3, partial_stride=sh.stride(0),
                                  bias=bias.to(DEV) if with_bias else None, maps=2)
        assert int(status.item()) == 0
        tol = 1e-5 if dtype == "float32" else 8e-3
        assert rel_err(q_out, q.reshape(n, -1)) < tol
        pages = table[torch.tensor(positions) // page].long()
        slots = torch.tensor(positions) % page
        assert rel_err(cache.k_pool[pages, :, slots], k.reshape(n, G, 2 * d)) < tol
        assert rel_err(cache.v_pool[pages, :, slots], v) < tol


def paged_from(seqs, ks, vs, first_keys, *, page_size, dtype, seed=0):
    """Key rows [tokens, kv heads, d] and values of some sequences scattered over pages handed out in random order; slots
    never written hold NaN, and pages wholly below a sequence's first key do not exist (they have been given back)."""
    from flambeau_b200.cache.manager import LayerCacheView
    g = torch.Generator().manual_seed(seed)
    G, d, e = ks[0].shape[1], ks[0].shape[2], vs[0].shape[2]
    first = [key // page_size for key in first_keys]
    count = [-(-(ctx + n) // page_size) for ctx, n in seqs]
    order = torch.randperm(sum(count) + 3, generator=g).tolist()
    table = torch.full((len(seqs), max(c - f for c, f in zip(count, first)) + 1), -1, dtype=torch.int32)
    k_pool = torch.full((sum(count) + 3, G, page_size, d), float("nan"), dtype=dtype)
    v_pool = torch.full((sum(count) + 3, G, page_size, e), float("nan"), dtype=dtype)
    for s, (ctx, n) in enumerate(seqs):
        for j in range(first[s], count[s]):
            page = order.pop()
            table[s, j - first[s]] = page
            lo, hi = j * page_size, min((j + 1) * page_size, ctx + n)
            k_pool[page, :, :hi - lo] = ks[s][lo:hi].transpose(0, 1).to(dtype)
            v_pool[page, :, :hi - lo] = vs[s][lo:hi].transpose(0, 1).to(dtype)
    return LayerCacheView(k_pool.to(DEV), v_pool.to(DEV), table.to(DEV), i32(first), page_size, False, 0, None)


# (heads, kv heads, key size per map, value size, chunk, page size)
CHUNKED = [(4, 2, 16, 48, 20, 16), (6, 1, 16, 32, 33, 16), (8, 2, 48, 64, 100, 16), (2, 1, 64, 128, 40, 8), (20, 1, 16, 16, 12, 16),
           (4, 1, 32, 80, 64, 16), (2, 2, 128, 256, 48, 32), (3, 3, 8, 20, 5, 16), (1, 1, 16, 16, 1, 16), (6, 3, 48, 96, 70, 16),
           (4, 4, 32, 64, 16, 16), (2, 1, 64, 64, 256, 64), (4, 2, 128, 128, 31, 16), (3, 1, 10, 18, 17, 16)]


@pytest.mark.parametrize("geometry", CHUNKED, ids=lambda g: "h%d.%d-k%d-v%d-c%d-p%d" % g)
@pytest.mark.parametrize("window", [0, 23])
@pytest.mark.parametrize("kernel", ["simt-float32", "simt-bfloat16", "mma-bfloat16"])
def test_differential_attention_within_chunks(geometry, window, kernel):
    """First tokens, positions at the ends of chunks, decoded tokens far into a request and at page borders, portions that
    cross a chunk's edge or several, portions of two tokens on either side of it; pages of chunks that were left are given
    back and unreadable.  For the first and last query of every sequence the chunk's first key stands out along both maps'
    queries and the key just below the chunk (which must not be seen) stands out more."""
    from flambeau_b200.kernels import ops
    nh, nkv, kd, vd, chunk, page = geometry
    which, dtype = kernel.split("-")
    dt = DT[dtype]
    c2 = 2 * chunk
    seqs = [(0, 1), (0, 37), (chunk - 1, 1), (chunk, 1), (c2 - 1, 2), (c2, 2), (c2 + 1, 3), (199, 1), (page * 3 - 1, 1),
            (page * 3, 1), (page * 2 + 5, 29), (63, 70), (10, 300), (5 * chunk - 1, 1), (max(0, c2 - 3), 17)]
    g = torch.Generator().manual_seed(nh * 100 + kd)
    scale, lam, diff, eps = 0.3, 0.62, 0.35, 1e-5
    group = torch.arange(nh) // (nh // nkv)
    qs, ks, vs, firsts, want = [], [], [], [], []
    for ctx, n in seqs:
        T = ctx + n
        q, k, v = (torch.randn(*s, generator=g).to(dt).double() for s in ((n, nh, 2, kd), (T, nkv, 2, kd), (T, nkv, vd)))
        for row in (0, n - 1):
            start = (ctx + row) // chunk * chunk
            for at, strength in ((start, 12.0), (start - 1, 40.0)):
                if at >= 0:
                    unit = q[row, 0] / (q[row, 0] ** 2).sum(-1, keepdim=True)
                    k[at, 0] = (unit * strength / scale).to(dt).double()
        i, j = torch.arange(ctx, T)[:, None], torch.arange(T)[None, :]
        seen = (j <= i) & (i // chunk == j // chunk)
        if window:
            seen = seen & (i - j < window)
        a = [torch.einsum("hij,jhe->ihe", ps.masked_softmax(torch.einsum("ihd,jhd->hij", q[:, :, m], k[:, group, m]) * scale,
                                                            seen[None]), v[:, group]) for m in (0, 1)]
        want.append(ps.difference_of_maps(a[0], a[1], lam, diff, eps))
        firsts.append(int(seen[0].nonzero()[0]))
        qs.append(q), ks.append(k.view(T, nkv, 2 * kd)), vs.append(v)
    cache = paged_from(seqs, ks, vs, firsts, page_size=page, dtype=dt)
    lens = [n for _, n in seqs]
    q_d = torch.cat([q.reshape(q.shape[0], -1) for q in qs]).to(dt).to(DEV)
    out, status = torch.full((sum(lens), nh * vd), float("nan"), dtype=dt, device=DEV), i32([0])
    if which == "mma":
        if not ops.diff_attention_mma_supported(q_d, nh, nkv, kd, vd):
            pytest.skip("sizes the tensor-core arrangements do not take run on the float32-math kernel")
        short = [n * (nh // nkv) <= 16 for n in lens]
        ops.diff_attention_mma(q_d, out, None, cache, i32([sum(lens[:i]) for i in range(len(lens))]), i32(lens),
                               i32([c for c, _ in seqs]), len(seqs), max(lens), max(c + n for c, n in seqs), any(short),
                               not all(short), nh, nkv, kd, vd, window, scale, lam, eps, 1.0 - diff, status, chunk=chunk)
    else:
        ops.diff_attention_simt(q_d, out, None, cache, i32([p for c, n in seqs for p in range(c, c + n)]),
                                i32([s for s, n in enumerate(lens) for _ in range(n)]), nh, nkv, kd, vd, window, scale, lam, eps,
                                1.0 - diff, status, chunk=chunk)
    assert int(status.item()) == 0 and bool(torch.isfinite(out.float()).all())
    assert rel_err(out, torch.cat(want).reshape(sum(lens), -1)) < (2e-5 if dtype == "float32" else 8e-3)


@pytest.mark.parametrize("shape", [(1, 12, 40, 5, 33), (9, 24, 96, 24, 144), (64, 128, 128, 128, 128), (130, 16, 70, 66, 64), (700, 8, 200, 12, 17)],
                         ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_maps_through_narrow_middles(shape, dtype):
    """Both maps of a launch with widths of their own, one alone, every function; middles that start on any column."""
    from flambeau_b200.kernels import ops
    n, R1, N1, R2, N2 = shape
    dt = DT[dtype]
    g = torch.Generator().manual_seed(n)
    group = 7
    for first in (0, 3, 8):
        pad = -(-(first + R1 + R2 + 2) // 8) * 8
        shares = torch.randn(3, n, pad, generator=g) * 0.6
        z = shares.double().sum(0)
        if dtype == "bfloat16":
            z = z.float().bfloat16().double()            # the middle is rounded once
        w1, w2 = (torch.randn(N, R, generator=g).to(dt) * 0.5 for N, R in ((N1, R1), (N2, R2)))
        bias, rate = (torch.randn(k, generator=g).to(dt) for k in (N1, -(-N1 // group)))
        y1 = z[:, first:first + R1] @ w1.double().T + bias.double()
        y2 = z[:, first + R1:first + R1 + R2] @ w2.double().T
        decay = torch.exp(-torch.exp(rate.double())[torch.arange(N1) // group] * ps.softplus(y1))
        sh = shares.to(DEV)
        for functions, want in ((("decay", "plain"), (decay, y2)), (("plain", "sigmoid"), (y1, torch.sigmoid(y2))), (("sigmoid",), (torch.sigmoid(y1),))):
            outs = [torch.full((n, N), float("nan"), device=DEV) for N in (N1, N2)]
            maps = [ops.LowRankMap(w1.to(DEV), first, outs[0], functions[0], bias=bias.to(DEV), log_rate=rate.to(DEV), group=group)]
            if len(functions) == 2:
                maps.append(ops.LowRankMap(w2.to(DEV), first + R1, outs[1], functions[1]))
            ops.low_rank_maps(sh[0], maps, n_partials=3, partial_stride=sh.stride(0))
            for out, ref in zip(outs, want):
                # (a middle on the border between two bfloat16 numbers may be rounded to either)
                assert float((out.double().cpu() - ref).abs().max()) / max(1.0, float(ref.abs().max())) < (5e-6 if dtype == "float32" else 4e-3)


@pytest.mark.parametrize("sizes", [(4, 2, 8, 16, 4), (2, 1, 16, 24, 3), (3, 3, 24, 8, 2), (2, 2, 40, 12, 1), (1, 1, 136, 72, 4),
                                   (4, 1, 300, 20, 2), (2, 1, 64, 128, 4), (2, 1, 128, 128, 4), (3, 1, 10, 6, 3), (1, 1, 513, 4, 2)], ids=str)
def test_delta_rule_with_a_decay_per_channel_across_steps(sizes):
    """Three requests in three state slots, fed in steps of unequal portions (one token, two tokens, many), then a slot
    zeroed and used again; the outputs of every step against the plain recurrence over the whole sequences.  Decays from
    nearly nothing to nearly all."""
    from flambeau_b200.kernels import ops
    H, G, dk, dv, taps = sizes
    g = torch.Generator().manual_seed(11)
    C, eps, lengths = 2 * G * dk + H * dv, 1e-5, [23, 9, 108]
    cols = -(-(C + H + 3) // 4) * 4
    conv_w, norm_w = torch.randn(C, taps, generator=g) * 0.5, torch.randn(dv, generator=g) + 1
    proj = [torch.randn(L, cols, generator=g) for L in lengths]
    decays = [torch.sigmoid(torch.randn(L, H * dk, generator=g) * 3.0 + 1.0) for L in lengths]
    gates = [torch.randn(L, H * dv, generator=g) for L in lengths]

    def plain(x, dec, gate):
        n = x.shape[0]
        act = ps.silu(ps.short_convolution(x.double()[:, :C], conv_w.double()))
        q = ps.unit_vector(act[:, :G * dk].reshape(n, G, dk)) * dk ** -0.5
        k = ps.unit_vector(act[:, G * dk:2 * G * dk].reshape(n, G, dk))
        v = act[:, 2 * G * dk:].reshape(n, H, dv)
        beta, dec = torch.sigmoid(x.double()[:, C + 3:C + 3 + H]), dec.double().view(n, H, dk)
        heads = [ps.rms_norm(ps.delta_rule(q[:, hh // (H // G)], k[:, hh // (H // G)], v[:, hh], beta[:, hh], dec[:, hh]),
                             norm_w.double(), eps) for hh in range(H)]
        return torch.cat(heads, dim=-1) * torch.sigmoid(gate.double())
    want = [plain(*x) for x in zip(proj, decays, gates)]
    S = H * dk * dv
    state = torch.zeros((4, -(-(S + (taps - 1) * C) // 4) * 4), dtype=torch.float32, device=DEV)
    state[3].fill_(float("nan"))                     # a slot nobody uses
    slots = [2, 0, 1]

    def step(live, at):
        x, dec, gate = (torch.cat([t[s][at[s]:at[s] + k] for s, k in live]).to(DEV) for t in (proj, decays, gates))
        shares = torch.stack([x * 0.25, x * 0.75])
        n = x.shape[0]
        b = fake_batch([k for _, k in live], [slots[s] for s, _ in live])
        qkv, beta = torch.empty((n, C), device=DEV), torch.empty((n, H), device=DEV)
        ops.gdr_prepare(shares[0], conv_w.to(DEV), taps, None, None, state, S, b, qkv, beta, None, G, H, dk, dv, dk ** -0.5,
                        1e-6, n_partials=2, partial_stride=shares.stride(0), b_off=C + 3)
        o, out = torch.empty((n, H * dv), device=DEV), torch.empty((n, H * dv), device=DEV)
        ops.gdr_channel_recurrent(qkv, beta, dec.contiguous(), state, b, o, G, H, dk, dv)
        ops.gdr_out_norm(o, gate, 0, norm_w.to(DEV), eps, out, H, dv, gate="sigmoid")
        as_is = torch.empty_like(out)
        ops.gdr_out_norm(o, torch.sigmoid(gate), 0, norm_w.to(DEV), eps, as_is, H, dv, gate=None)
        assert rel_err(as_is, out.double().cpu()) < 1e-5
        return out.cpu()
    at, got = [0, 0, 0], [[], [], []]
    for portion in [[1, 2, 5], [2, 1, 17], [3, 0, 1], [16, 6, 84], [1, 0, 1]]:
        live = [(s, k) for s, k in enumerate(portion) if k]
        out, r = step(live, at), 0
        for s, k in live:
            got[s].append(out[r:r + k])
            r, at[s] = r + k, at[s] + k
    assert at == lengths
    for s in range(3):
        assert rel_err(torch.cat(got[s]), want[s]) < 3e-5
    state[slots[1]].zero_()                          # given back and used again: it starts from zero once more
    assert rel_err(step([(1, lengths[1])], [0, 0, 0]), want[1]) < 3e-5
    assert bool(torch.isnan(state[3]).all()), "a slot that no sequence of the step uses was written"


# ---------------------------------------------------------------------------------------------------------------
# parts alone, through the step context, cache and state slots the engine uses
# ---------------------------------------------------------------------------------------------------------------
def mixer_in_steps(layer, dtype, width=48, eps=1e-5, redraw=()):
    """The mixer of a layer as the model builds it, run over STEPS; (got, oracle's output) per request.  redraw: (leaf,
    std, centre) of tensors that are drawn anew."""
    from test_parts_gpu import Bench
    from flambeau_b200 import models  # noqa: F401
    from flambeau_b200.cache.manager import CallPlan
    from flambeau_b200.config.sisadra import MIXERS
    from flambeau_b200.config.base import ConfigReader
    from flambeau_b200.models.sisadra import _mixer
    from flambeau_b200.parts.spec import build_part
    from flambeau_b200.weights.random_init import draw
    m = MIXERS[layer["type"]].from_reader(ConfigReader(layer["mixer"]), "m")
    spec = _mixer(layer["type"], m, width, eps, "m.")
    probe = build_part(spec, None)
    b = Bench(dtype, plans=[CallPlan(kv=probe.cache_requirement(), state=probe.state_requirement())])
    part = build_part(spec, b.rt)
    g = torch.Generator().manual_seed(2)
    W = {}
    for name, ts in part.tensor_specs().items():
        t = draw(ts, 0, name)
        std, centre = next(((s, c) for leaf, s, c in redraw if name.endswith(leaf)), (0.15, 0.0) if t.dim() == 2 else (None, 0.0))
        W[name] = ((torch.randn(ts.shape, generator=g) * std + centre) if std is not None else t).to(DT[dtype])
    part.bind({k: v.to(DEV) for k, v in W.items()})
    Hs = {"a": torch.randn(174, width, generator=g).to(DT[dtype]), "b": torch.randn(24, width, generator=g).to(DT[dtype])}
    got = run_mixer_in_steps(b, part, Hs, STEPS, width)
    W = {k: v.double() for k, v in W.items()}
    return {rid: (got[rid], ps.MIXERS[layer["type"]](h.double(), W, "m.", layer["mixer"], eps)) for rid, h in Hs.items()}


@pytest.mark.parametrize("layer", [st.attention(4, 2, 32, 48, 20, st.rotation(1e4, 8, 3.0)), st.attention(6, 1, 16, 16, 7),
                                   st.attention(3, 3, 10, 18, 16, st.rotation(300.0, 10)), st.attention(2, 1, 64, 128, 1, st.rotation(1e3, 64, 2.0)),
                                   st.attention(5, 5, 48, 96, 0, st.rotation(2e5, 32, 6.0, 1.0, 5.0, 40)), st.attention(18, 1, 16, 32, 64),
                                   st.attention(2, 2, 6, 10, 33, st.rotation(50.0, 2, 4.0))], ids=lambda l: "-".join(str(x) for x in l["mixer"].values() if isinstance(x, int)))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_differential_attention_part(layer, dtype):
    """Norms with weights far from one, biases that matter on all four maps, over steps of portions and single tokens."""
    redraw = [(".norm", 0.6, 1.5), ("o.b", 1.0, 0.0), (".b", 0.4, 0.0), ("lq1", 0.4, 0.0), ("lk1", 0.4, 0.0)]
    for rid, (got, want) in mixer_in_steps(layer, dtype, redraw=redraw).items():
        assert rel_err(got, want) < (2e-5 if dtype == "float32" else 2e-2), rid


@pytest.mark.parametrize("layer", [st.latent(3, 16, 24, 48), st.latent(18, 8, 16, 80), st.latent(2, 6, 10, 20), st.latent(1, 32, 8, 256),
                                   st.latent(5, 12, 12, 12), st.latent(20, 16, 16, 64, 0.1)], ids=lambda l: "-".join(str(x) for x in l["mixer"].values() if isinstance(x, int)))
@pytest.mark.parametrize("sink", [-3.0, 4.0])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_attention_part_with_a_sink(layer, sink, dtype):
    """A sink that takes hardly anything, and one that takes most of a softmax over few keys."""
    redraw = [("sink", 0.5, sink), (".norm", 0.4, 1.0)]
    for rid, (got, want) in mixer_in_steps(layer, dtype, redraw=redraw).items():
        assert rel_err(got, want) < (2e-5 if dtype == "float32" else 2e-2), rid


@pytest.mark.parametrize("layer", [st.delta(6, 2, 24, 16, 4), st.delta(3, 3, 16, 32, 1), st.delta(4, 2, 40, 72, 2), st.delta(3, 1, 10, 6, 3),
                                   st.delta(2, 1, 128, 64, 4), st.delta(2, 2, 64, 64, 5)], ids=lambda l: "-".join(str(x) for x in l["mixer"].values()))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_channel_delta_part(layer, dtype):
    redraw = [("A_log", 1.0, -1.5), ("a2", 0.4, 0.0), ("g2", 0.4, 0.0), (".norm", 0.4, 1.0), (".conv", 0.4, 0.0)]
    for rid, (got, want) in mixer_in_steps(layer, dtype, redraw=redraw).items():
        assert rel_err(got, want) < (5e-5 if dtype == "float32" else 2e-2), rid


@pytest.mark.parametrize("n,width,ff", [(1, 64, 48), (5, 96, 48), (64, 256, 512), (300, 72, 64), (600, 256, 512), (40, 50, 30)])
@pytest.mark.parametrize("with_mlp", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_an_attention_layer_whose_output_bias_joins_the_stream(tmp_path, n, width, ff, with_mlp, dtype):
    """Logits of one-layer models at sizes where the output projection leaves shares, one share, or adds to the stream by
    itself, and with the bias left to the feed-forward's norm or added on its own; biases that outweigh the rest."""
    cfg = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 100, "width": width, "embedding": {"scale": 1.0},
           "layers": [dict(st.attention(3, 1, 16, 16, 30), mlp=st.dense(ff) if with_mlp else None)]}
    c = make_case(f"bias {n}x{width}", cfg, tmp_path / "m", dtype, [n], seed=n)
    tensors = st.read_tensors(c["folder"])
    tensors["l0.mix.o.b"] = (torch.randn(width, generator=torch.Generator().manual_seed(1)) * 2.0).to(DT[dtype])
    st.write_tensors(c["folder"], tensors)
    pcfg, W = ps.read_folder(c["folder"])
    c["want"] = {rid: ps.forward(pcfg, W, toks) for rid, toks in c["requests"].items()}
    run(c, tiny.schedule_whole(c["requests"]), tmp_path / "o")


# ---------------------------------------------------------------------------------------------------------------
# whole models under schedules
# ---------------------------------------------------------------------------------------------------------------
SHARP = {"float32": 0.25, "bfloat16": 0.12}
LENGTHS = {"DA": [1, 9, 40, 75, 33, 21, 64, 110], "DB": [2, 70, 17, 48, 150, 5], "DC": [30, 3, 50]}


def tolerance(dtype, pcfg, W, requests):
    """(bound on the worst position, bound on the median position), as fractions of the logit scale.  float32: 1e-4
    for both.  bfloat16: three times what rounding alone causes, which the plain implementation measures on the same
    requests by rounding the values a 16-bit engine keeps in 16 bits; never below the 2e-2 and a quarter of it that fit
    the framework's other models."""
    if dtype == "float32":
        return 1e-4, 1e-4
    noise = [ps.rounding_noise(pcfg, W, toks) for toks in requests.values()]
    worst, median = max(w for w, _ in noise), max(m for _, m in noise)
    return max(tiny.TOL["bfloat16"], 3.0 * worst), max(tiny.TOL["bfloat16"] / 4, 3.0 * median)


def make_case(name, cfg, folder, dtype, lengths, seed, request_seed=4):
    st.make_folder(folder, cfg, seed=seed, dtype=dtype, sharp=SHARP[dtype])
    requests = tiny.random_requests({"vocab_size": cfg["vocab"]}, lengths, seed=request_seed)
    pcfg, W = ps.read_folder(folder)
    want = {rid: ps.forward(pcfg, W, toks) for rid, toks in requests.items()}
    return dict(name=name, dtype=dtype, cfg=cfg, folder=folder, requests=requests, want=want,
                tol=tolerance(dtype, pcfg, W, requests))


@pytest.fixture(scope="module", params=[(c, d) for c in ("DA", "DB") for d in ("float32", "bfloat16")],
                ids=lambda p: f"{p[0]}-{p[1]}")
def case(request, tmp_path_factory):
    name, dtype = request.param
    return make_case(name, st.CONFIGS[name], tmp_path_factory.mktemp(f"s{name}{dtype}"), dtype, LENGTHS[name],
                     seed=17 if name == "DA" else 29)


def run(case, schedule, out_dir, cuda_graphs=True):
    from flambeau_b200.engine.step import Engine, EngineOptions
    from flambeau_b200.engine.trace import replay
    tokens = schedule.max_live_tokens(case["requests"])
    engine = Engine.from_folder(case["folder"], EngineOptions(
        dtype=case["dtype"], cache_tokens=tokens, max_requests=4, max_step_tokens=max(tokens, 128),
        max_seq_len=max(tokens, 192), cuda_graphs=cuda_graphs))
    replay(engine, schedule.lines(), out_dir)
    run.last_engine = engine
    engine.cache.check_invariants()
    assert not engine.cache.requests, "requests left live after the trace"
    assert all(g.pool.n_free == g.pool.n_pages for g in engine.cache.groups), "pages lost"
    got = tiny.read_rows(out_dir, schedule, case["cfg"]["vocab"])
    return compare(got, case["want"], case["tol"], f"{case['name']} {case['dtype']}")


def test_whole(case, tmp_path):
    run(case, tiny.schedule_whole(case["requests"]), tmp_path)


def test_last_tokens_one_by_one_past_the_chunks(case, tmp_path):
    """The tail is longer than most of the chunks, so decoded tokens leave chunks behind and give pages back."""
    run(case, tiny.schedule_tail(case["requests"], 45), tmp_path)


def test_portions_down_to_two_tokens(case, tmp_path):
    run(case, tiny.schedule_portions(case["requests"]), tmp_path)
    run(case, tiny.schedule_portions(case["requests"], sizes=(2, 31, 2, 2, 17, 64, 3)), tmp_path / "b")


@pytest.mark.parametrize("seed", [1, 2])
def test_mixed_batches_with_pages_and_slots_used_again(case, tmp_path, seed):
    sched = tiny.schedule_mixed(case["requests"], seed=seed)
    total_pages = sum(-(-len(t) // 16) for t in case["requests"].values())
    assert sched.max_live_tokens(case["requests"]) // 16 < total_pages, "the pool must be smaller than all requests"
    assert len(case["requests"]) > 4, "more requests than slots, so that slots are used again"
    run(case, sched, tmp_path)


def test_every_token_decoded_from_the_first(case, tmp_path):
    """One token a step from position 0 (replayed from CUDA graphs where the engine captures them): the first tokens
    of a sequence, and a long decoding."""
    rid = max(case["requests"], key=lambda r: len(case["requests"][r]))
    toks = case["requests"][rid]
    s = tiny.Schedule()
    for p, t in enumerate(toks):
        s.add([(rid, [t], [0], p)], end=[rid] if p == len(toks) - 1 else [])
    one = dict(case, requests={rid: toks}, want={rid: case["want"][rid]})
    run(one, s, tmp_path)
    assert run.last_engine.graph_replays > len(toks) // 2, "single-token steps are replayed from a captured graph"


def test_ids_used_again_and_requests_ended_early(case, tmp_path):
    """A trace as a careless client writes it (tiny.schedule_wild): what a slot holds (states, tails, the token before) must
    not reach the next request that gets the slot."""
    from flambeau_b200.engine.step import Engine, EngineOptions
    from flambeau_b200.engine.trace import replay
    for seed in (3, 4):
        requests, sched = tiny.schedule_wild({"vocab_size": case["cfg"]["vocab"]}, seed=seed)
        pcfg, W = ps.read_folder(case["folder"])
        engine = Engine.from_folder(case["folder"], EngineOptions(dtype=case["dtype"], cache_tokens=1024, max_requests=4,
                                                                  max_step_tokens=512))
        replay(engine, sched.lines(), tmp_path / str(seed))
        got = tiny.read_rows(tmp_path / str(seed), sched, case["cfg"]["vocab"])
        full = {u: ps.forward(pcfg, W, toks).numpy() for u, toks in requests.items() if any(k[0] == u for k in got)}
        for (u, p), row in got.items():
            err = abs(row - full[u][p]).max() / abs(full[u]).max()
            assert err <= case["tol"][0], (seed, u, p, err)


def test_odd_sizes(tmp_path):
    for dtype in ("float32", "bfloat16"):
        c = make_case("DC", st.CONFIGS["DC"], tmp_path / dtype, dtype, LENGTHS["DC"], seed=3, request_seed=2)
        run(c, tiny.schedule_portions(c["requests"], sizes=(5, 2, 9)), tmp_path / dtype / "o")
        run(c, tiny.schedule_tail(c["requests"], 12), tmp_path / dtype / "t")


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: widths that are and are not multiples of 8, odd head sizes, chunks from one key
    to beyond the requests, scaled and plain rotations of part of a map, latents of any size, one to five taps, with and
    without a pair table, a cap, feed-forwards."""
    import random
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(2, 5)):
        heads, kv = rng.choice([(1, 1), (2, 1), (4, 2), (6, 3), (3, 3), (18, 1)])
        d, e = rng.choice([6, 8, 16, 24, 32, 48]), rng.choice([8, 10, 16, 32, 64])
        kind = rng.choice(["attention", "latent", "delta"])
        if kind == "attention":
            rot = rng.choice([None, st.rotation(rng.choice([100.0, 1e4, 5e5]), rng.choice([2, d]), rng.choice([None, 2.0, 8.0]),
                                                rng.choice([1.0, 0.5]), rng.choice([2.0, 4.0, 30.0]), rng.choice([16, 100, 1024]))])
            mix = st.attention(heads, kv, d, e, rng.choice([0, 1, 2, 5, 16, 17, 31, 64, 500]), rot, rng.uniform(0.1, 0.4), rng.uniform(0.1, 0.8))
        elif kind == "latent":
            mix = st.latent(heads, d, e, rng.choice([8, 20, 36, 64, 128]), rng.uniform(0.1, 0.4))
        else:
            mix = st.delta(heads, kv, d, e, rng.randint(1, 5))
        layers.append(dict(mix, mlp=st.dense(rng.choice([24, 40, 100])) if rng.random() < 0.6 else None))
    cfg = {"architecture": "Sisadra", "norm": {"eps": rng.choice([1e-5, 1e-6])}, "vocab": rng.randint(50, 400),
           "width": rng.choice([40, 72, 100, 128, 36]), "layers": layers, "embedding": {"scale": rng.choice([0.5, 1.0, 4.0])}}
    if rng.random() < 0.7:
        cfg["embedding"]["bigram"] = st.bigram(rng.choice([1, 7, 100, 1009]), rng.randint(1, 10 ** 6), rng.randint(1, 10 ** 6))
    if rng.random() < 0.7:
        cfg["logit_softcap"] = rng.uniform(3.0, 40.0)
    return cfg


@pytest.mark.parametrize("seed", [501, 502, 503, 504, 505, 506, 507, 508, 509, 510])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configurations_under_a_mixed_schedule(tmp_path, seed, dtype):
    c = make_case(f"random {seed}", random_config(seed), tmp_path / "m", dtype, [1, 37, 80, 2, 55, 21], seed=seed, request_seed=seed)
    run(c, tiny.schedule_mixed(c["requests"], seed=seed), tmp_path / "o")


def logits_at_the_end(folder, tokens, cut, dtype="float32"):
    """The last position's logits, the request fed as tokens[:cut] and then the rest (a single token when cut is
    len - 1: the position is then a decoded one)."""
    from flambeau_b200.engine.step import Engine, EngineOptions
    engine = Engine.from_folder(folder, EngineOptions(dtype=dtype, cache_tokens=1024, max_requests=2, max_step_tokens=512))
    if cut:
        engine.step([("a", tokens[:cut], [])])
    return engine.step([("a", tokens[cut:], [len(tokens) - cut - 1])], end=["a"])[0].double().cpu()


@pytest.mark.parametrize("chunk,length", [(1, 60), (2, 77), (11, 96), (16, 80), (16, 81), (17, 120), (64, 128), (64, 129), (70, 160)])
def test_chunks_end_where_they_should_in_prompts_and_in_decoding(tmp_path, chunk, length):
    """One layer without feed-forward and without pairs, float32: a token then reaches later positions through its key and
    value alone.  Changing the token just below the last query's chunk leaves its logits as they were; changing the
    chunk's first token moves them.  The last position is once part of a portion, once a decoded token; it is the chunk's
    last, its first, or in its middle."""
    cfg = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 150, "width": 48, "embedding": {"scale": 1.0},
           "layers": [dict(st.attention(3, 1, 16, 24, chunk, st.rotation(1e4, 8, 2.0)), mlp=None)]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=8, dtype="float32", sharp=0.12)
    base = tiny.random_requests({"vocab_size": cfg["vocab"]}, [length], seed=1)["r0"]
    p = length - 1
    start = p // chunk * chunk

    def moves(at, cut, ref):
        t = list(base)
        t[at] = (t[at] + 1) % cfg["vocab"]
        return float((logits_at_the_end(folder, t, cut) - ref).abs().max()) / float(ref.abs().max())
    for cut in (length // 3, p - 1, p):              # (p: the last token is decoded alone)
        ref = logits_at_the_end(folder, base, cut)
        assert moves(start - 1, cut, ref) < 1e-6, cut
        if start < p:
            assert moves(start, cut, ref) > 1e-5, cut
    pcfg, W = ps.read_folder(folder)
    assert rel_err(logits_at_the_end(folder, base, 37), ps.forward(pcfg, W, base)[-1]) < 1e-4


def test_the_state_carries_a_far_token_and_a_freed_slot_forgets_it(tmp_path):
    """One recurrent layer with slow decays, float32: a token hundreds of positions back still moves the last logits (the
    state has carried it, through portions and single tokens); a second request in the slot the first one gave back, and
    one that comes back from a snapshot into another slot, get the logits of a request that runs alone."""
    from flambeau_b200.engine.step import Engine, EngineOptions
    cfg = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 150, "width": 48,
           "embedding": {"scale": 1.0, "bigram": st.bigram(1009, 31, 7)},
           "layers": [dict(st.delta(4, 2, 16, 24, 4), mlp=st.dense(40))]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=9, dtype="float32")
    tensors = st.read_tensors(folder)
    tensors["l0.mix.A_log"][:] = -7.0
    st.write_tensors(folder, tensors)
    base = tiny.random_requests({"vocab_size": cfg["vocab"]}, [300], seed=2)["r0"]
    other = list(base)
    other[3] = (other[3] + 1) % cfg["vocab"]
    ref = logits_at_the_end(folder, base, 280)
    assert float((logits_at_the_end(folder, other, 299) - ref).abs().max()) / float(ref.abs().max()) > 1e-4
    pcfg, W = ps.read_folder(folder)
    assert rel_err(ref, ps.forward(pcfg, W, base)[-1]) < 1e-4
    engine = Engine.from_folder(folder, EngineOptions(dtype="float32", cache_tokens=1024, max_requests=2, max_step_tokens=512))
    engine.step([("a", other, [])], end=["a"])
    engine.step([("b", base[:200], [])])
    kept = engine.snapshot("b")
    engine.finish("b")
    engine.step([("y", other[:40], []), ("z", [4], [])], end=["y"])
    engine.restore("b", kept)
    engine.step([("b", base[200:299], []), ("z", [5], [])])
    again = engine.step([("z", [6], []), ("b", base[299:], [0])])[0].double().cpu()
    assert float((again - ref).abs().max()) / float(ref.abs().max()) < 1e-5


def test_the_token_before_is_kept_from_step_to_step(tmp_path):
    """Chunks of one key: the token before reaches a position through the pair table alone.  It moves the logits however the
    request is cut, the one before it does not; a first token takes the row of its own whatever the slot held."""
    from flambeau_b200.engine.step import Engine, EngineOptions
    cfg = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 60, "width": 32,
           "embedding": {"scale": 3.0, "bigram": st.bigram(1009, 31, 7)}, "layers": [dict(st.attention(2, 1, 16, 16, 1), mlp=None)]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=4, dtype="float32")
    pcfg, W = ps.read_folder(folder)
    base = [5, 9, 11, 3, 40, 22]
    want = ps.forward(pcfg, W, base)
    for cut in range(len(base)):
        assert rel_err(logits_at_the_end(folder, base, cut), want[-1]) < 1e-4, cut
    assert rel_err(logits_at_the_end(folder, base[:4] + [41, 22], 5), want[-1]) > 1e-2
    assert rel_err(logits_at_the_end(folder, base[:3] + [8, 40, 22], 5), want[-1]) < 1e-4
    engine = Engine.from_folder(folder, EngineOptions(dtype="float32", cache_tokens=512, max_requests=2, max_step_tokens=64))
    for rid in ("a", "b", "c", "d"):                 # slots used again
        first = engine.step([(rid, [22], [0])])[0].double().cpu()
        assert rel_err(first, ps.forward(pcfg, W, [22])[0]) < 1e-4, rid
        engine.step([(rid, [7, 8], [])], end=[rid])


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_a_far_key_among_hundreds_is_found(tmp_path, kind):
    """No mask, float32: one head's maps are rebuilt so that its query for one token points along another token's key (or
    latent).  Where the first stands last and the second hundreds of positions back and nowhere else, that far key takes
    most of the head's softmax, so that losing the key, or its page, would move the logits by far more than rounding."""
    mix = st.attention(2, 1, 16, 16, 0, st.rotation(1e4, 4, 2.0), 1.0) if kind == "attention" else st.latent(2, 8, 8, 16, 1.0)
    cfg = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 90, "width": 32, "embedding": {"scale": 1.0},
           "layers": [dict(mix, mlp=None)]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=10, dtype="float32", sharp=0.3)
    _, W = ps.read_folder(folder)
    asks, answers = 85, 84
    h = ps.centred_norm(W["embed"][[asks, answers]], W["l0.norm1"], 1e-5)
    point = (8.0 * h / (h ** 2).sum(-1, keepdim=True)).float()      # 8 along each of the two tokens' normed rows
    t = st.read_tensors(folder)
    if kind == "attention":
        for name in ("q.b", "k.b"):
            t["l0.mix." + name][:] = 0.0
        t["l0.mix.q.norm"][:], t["l0.mix.k.norm"][:] = 1.5, 1.0
        t["l0.mix.k"][8] = point[1]                  # map 1 of the one key head: dimension 8 (unrotated)
        t["l0.mix.q"][:16] = 0.0                     # map 1 of query head 0
        t["l0.mix.q"][8] = point[0]
    else:
        c = ps.rms_norm(h[1:] @ W["l0.mix.dkv"].T, W["l0.mix.dkv.norm"], 1e-5)
        t["l0.mix.uk"][:8] = 0.0
        t["l0.mix.uk"][0] = (c[0] / c[0].norm()).float()
        t["l0.mix.q"][:8] = 0.0
        t["l0.mix.q"][0] = point[0]
    st.write_tensors(folder, t)
    pcfg, W = ps.read_folder(folder)
    base = tiny.random_requests({"vocab_size": 80}, [400], seed=3)["r0"]      # tokens from 80 on are kept for the far key
    far = list(base)
    far[7], far[-1] = answers, asks
    want = ps.forward(pcfg, W, far)[-1]
    for cut in (150, len(far) - 1):
        assert rel_err(logits_at_the_end(folder, far, cut), want) < 1e-4
    moved = list(far)
    moved[7] = 86
    assert float((ps.forward(pcfg, W, moved)[-1] - want).abs().max()) / float(want.abs().max()) > 2e-2, \
        "the far key does not matter in this model: the test would show nothing"


# ---------------------------------------------------------------------------------------------------------------
# generation through the entry point and the scheduler
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name,dtype", [("DA", "float32"), ("DB", "bfloat16"), ("DA", "bfloat16")])
def test_greedy_generation(tmp_path, name, dtype):
    from flambeau_b200 import generate
    cfg = st.CONFIGS[name]
    folder = st.make_folder(tmp_path / "m", cfg, seed=41, dtype=dtype, sharp=SHARP[dtype])
    pcfg, W = ps.read_folder(folder)
    prompts = list(tiny.random_requests({"vocab_size": cfg["vocab"]}, [3, 26, 50, 1, 12], seed=6).values())
    n_new = 10
    outs = generate(folder, prompts, max_tokens=n_new, temperature=0.0, dtype=dtype, prefill_chunk_tokens=16,
                    prefill_ubatch=40, inflight_slots=3)
    tol = tolerance("bfloat16", pcfg, W, {i: p for i, p in enumerate(prompts)})[0]
    for prompt, out in zip(prompts, outs):
        assert len(out) == n_new
        toks = list(prompt)
        for t in out:
            logits = ps.forward(pcfg, W, toks)[-1]
            best = float(logits.max())
            if dtype == "float32":
                assert t == int((logits == best).nonzero()[0]), "greedy token differs from the plain implementation"
            else:
                gap = float(best - logits[t]) / float(logits.abs().max())
                assert gap <= 2 * tol, f"token {t} is {gap:.3f} of the scale below the best logit"
            toks.append(t)


def test_command_line_infer_and_replay(tmp_path):
    """The programs a user runs: `flambeau infer` (greedy, float32: the tokens are the plain implementation's) and
    `bin/trace_run` fed two requests step by step (their last logits are the plain implementation's)."""
    import json
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    root = Path(__file__).resolve().parent.parent
    cfg = st.CONFIGS["DC"]
    folder = st.make_folder(tmp_path / "m", cfg, seed=12, dtype="float32")
    pcfg, W = ps.read_folder(folder)
    prompt = tiny.random_requests({"vocab_size": cfg["vocab"]}, [14], seed=3)["r0"]
    proc = subprocess.run([sys.executable, str(root / "bin" / "flambeau"), "infer", "--model", str(folder), "--max-tokens",
                           "4", "--dtype", "float32", "--prompt", ",".join(map(str, prompt))],
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    toks = list(prompt)
    for t in (int(t) for t in proc.stdout.strip().splitlines()[-1].split(",")):
        logits = ps.forward(pcfg, W, toks)[-1]
        assert t == int((logits == logits.max()).nonzero()[0])
        toks.append(t)
    other = tiny.random_requests({"vocab_size": cfg["vocab"]}, [9], seed=5)["r0"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompt[:6], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": prompt[6:13], "want": []},
                                     {"id": "b", "tokens": other[:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": other[8:], "want": [0]},
                                     {"id": "a", "tokens": prompt[13:], "want": [0]}], "end": ["a", "b"]}]
    proc = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out",
                           str(tmp_path / "o"), "--max-tokens", "128"], input="\n".join(json.dumps(x) for x in steps) + "\n",
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4").reshape(2, cfg["vocab"])
    for row, seq in zip(got, (other, prompt)):
        assert rel_err(torch.from_numpy(row.copy()), ps.forward(pcfg, W, seq)[-1]) < 1e-4
