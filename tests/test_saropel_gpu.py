"""Saropel on the GPU against the plain implementation (tests/plain_saropel.py): each mechanism alone through its
kernels and parts, then whole models under schedules (whole, token by token, portions down to two tokens, mixed batches
on a pool so small that pages and slots are used again), the edges of windows in prompts and in decoding, the token
before across steps and slots, a far key among hundreds, long decoding, random configurations, and greedy generation
through generate()."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_saropel as ps
import saropel_tiny as st
import tiny
from test_tubepel_gpu import STEPS, compare, i32, paged_keys_and_values, rel_err, run_mixer_in_steps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


# ---------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("shape", [(64, 40, 53), (50, 30, 1), (1024, 300, 1000)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_of_pairs_across_steps_and_slots(shape, dtype):
    """Entries of several requests in one step, portions and single tokens, requests that sit out: the token before comes
    from the step or from the request's slot; a slot that was zeroed starts a request over."""
    from flambeau_b200.kernels import ops
    width, vocab, buckets = shape
    g = torch.Generator().manual_seed(width)
    dt = DT[dtype]
    E, P = torch.randn(vocab, width, generator=g).to(dt), torch.randn(buckets + 1, width, generator=g).to(dt)
    big = dict(buckets=buckets, mul_prev=1000003, mul_cur=-77)
    seqs = {s: torch.randint(0, vocab, (40,), generator=g).tolist() for s in range(3)}
    state = torch.zeros(4, 1, dtype=torch.int32, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    at = {s: 0 for s in seqs}
    slot_of = {0: 2, 1: 0, 2: 3}
    for step in ([(0, 1)], [(1, 7), (0, 3)], [(0, 1), (1, 1), (2, 2)], [(2, 30), (0, 1)], [(1, 2), (2, 1)], [(0, 9)]):
        ids = [t for s, k in step for t in seqs[s][at[s]:at[s] + k]]
        starts = [sum(k for _, k in step[:i]) for i in range(len(step))]
        batch = SimpleNamespace(row_seq=i32([i for i, (_, k) in enumerate(step) for _ in range(k)]), seq_q_start_d=i32(starts),
                                seq_q_len_d=i32([k for _, k in step]), seq_slot_d=i32([slot_of[s] for s, _ in step]))
        x = torch.empty(len(ids), width, dtype=torch.float32, device=DEV)
        ops.embedding_pairs(E.to(DEV), P.to(DEV), big["mul_prev"], big["mul_cur"], i32(ids), batch, state, x, status, 0.5)
        want = torch.cat([E.double()[seqs[s][at[s]:at[s] + k]] * 0.5 + P.double()[ps.pair_rows(seqs[s][:at[s] + k], big)[at[s]:]]
                          for s, k in step])
        assert rel_err(x, want) < 1e-6
        for s, k in step:
            at[s] += k
            assert int(state[slot_of[s]]) == seqs[s][at[s] - 1] + 1
    state[2].zero_()                                   # slot 2 goes to a new request
    batch = SimpleNamespace(row_seq=i32([0]), seq_q_start_d=i32([0]), seq_q_len_d=i32([1]), seq_slot_d=i32([2]))
    ops.embedding_pairs(E.to(DEV), P.to(DEV), 5, 7, i32([3]), batch, state, x[:1], status, 1.0)
    assert rel_err(x[:1], (E.double()[3] + P.double()[buckets])[None]) < 1e-6 and int(status.item()) == 0
    ops.embedding_pairs(E.to(DEV), P.to(DEV), 5, 7, i32([vocab]), batch, state, x[:1], status, 1.0)
    assert int(status.item()) == 1, "an id outside the table is flagged, not read"


@pytest.mark.parametrize("shape", [(5, 12, 16, 3), (70, 16, 16, 1), (33, 100, 104, 8)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gate_of_a_token_input(shape, dtype):
    from flambeau_b200.kernels import ops
    n, dim, cols, parts = shape
    g = torch.Generator().manual_seed(n)
    z = torch.randn(parts, n, cols + 4, generator=g) * 2.0
    table = torch.randn(50, 3 * dim, generator=g).to(DT[dtype])
    ids = torch.randint(0, 50, (n,), generator=g).tolist()
    out = torch.full((n, cols), 9.0, dtype=DT[dtype], device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.token_gate(z.to(DEV)[0], table.to(DEV), 2 * dim, dim, i32(ids), out, status, n_partials=parts,
                   partial_stride=z.stride(0))
    want = ps.gelu_tanh(z.double().sum(0)[:, :dim]) * table.double()[ids, 2 * dim:]
    assert rel_err(out[:, :dim], want) < (2e-6 if dtype == "float32" else 5e-3)
    assert bool((out[:, dim:] == 0).all()), "the padding columns are zeros"


@pytest.mark.parametrize("width", [64, 50, 4096])
def test_shares_join_the_stream_with_a_copy_and_rows_with_a_vector(width):
    from flambeau_b200.kernels import ops
    n = 19
    g = torch.Generator().manual_seed(width)
    x, d, y, v = (torch.randn(*s, generator=g) for s in ((n, width), (11, n, width), (n, width), (width,)))
    for dtype in DT.values():
        xd, dd, copy = x.to(DEV), d.to(DEV), torch.empty(n, width, dtype=dtype, device=DEV)
        ops.add_slabs(xd, dd[0], n, 11, dd.stride(0), copy=copy)
        want = x.double() + d.double().sum(0)
        assert rel_err(xd, want) < 1e-6 and torch.equal(copy, xd.to(dtype))
        ops.add_slabs(xd, None, n, copy=copy)
        assert rel_err(xd, want) < 1e-6 and torch.equal(copy, xd.to(dtype)), "nothing to add: the copy alone"
        for vec, rows in ((v, None), (None, y), (v, y)):
            xd = x.to(DEV)
            ops.add_row(xd, vec.to(dtype).to(DEV) if vec is not None else None, rows.to(DEV) if rows is not None else None)
            want = x.double() + (vec.to(dtype).double() if vec is not None else 0) + (rows.double() if rows is not None else 0)
            assert rel_err(xd, want) < 1e-6


@pytest.mark.parametrize("shape", [(5, 64, 24), (64, 96, 40), (130, 64, 80), (300, 128, 256), (600, 256, 512)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_feed_forward_with_cut_off_operands(shape, dtype):
    """Few rows (shares and the activation kernel) and many (the activation in the products' epilogues, one-SM and
    two-SM); inputs so large that both limits cut."""
    from test_parts_gpu import Bench, bind_random
    from flambeau_b200.parts.feedforward import GatedMLP
    n, D, ff = shape
    b = Bench(dtype, max_step_tokens=1024, cache_tokens=1024)
    part = GatedMLP(b.rt, "m.", width=D, inner=ff, activation="limited", limit=0.9, slope=1.702, init_std=0.2,
                    names=("gate", "up", "down"))
    Wt = bind_random(part, DT[dtype])
    h = torch.randn(n, D, generator=torch.Generator().manual_seed(n)).to(DT[dtype])
    z = h.double() @ Wt["m.gate"].T
    assert bool((z > 0.9).any()) and bool((h.double() @ Wt["m.up"].T < -0.9).any()), "nothing is cut off"
    ctx, _ = b.begin([("a", [1] * n, [])], D)
    ctx.pending_slabs = 1
    part.forward(ctx, h.to(DEV), ctx.delta)
    b.end()
    out = ctx.delta_slabs[:ctx.pending_slabs].sum(0)
    assert rel_err(out, ps.limited_expert(h.double(), Wt, "m.", 0.9)) < (2e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("experts", [(6, 3, 3, 2), (8, 2, 4, 1), (40, 5, 5, 2), (512, 8, 16, 3), (96, 6, 96, 7), (7, 3, 7, 7),
                                     (12, 4, 1, 1), (9, 9, 3, 3), (10, 4, 1, 0)], ids=str)
@pytest.mark.parametrize("renormalize", [False, True])
def test_router_chooses_within_the_best_groups(experts, renormalize):
    from flambeau_b200.kernels import ops
    E, K, count, keep = experts
    n, parts = 77, 3
    g = torch.Generator().manual_seed(E)
    z = torch.randn(parts, n, E + 9, generator=g) * 1.5
    chosen, share = torch.empty(n, K, dtype=torch.int32, device=DEV), torch.empty(n, K, device=DEV)
    gate = torch.empty(n, device=DEV)
    zd = z.to(DEV)
    ops.moe_choose(zd[0], None, E, E, K, chosen, share, gate, n_partials=parts, partial_stride=zd.stride(0),
                   rule="softmax_of_all", renormalize=renormalize, groups=count, keep_groups=keep)
    total = z.double().sum(0)
    router = {"top": K}
    if keep:
        router["groups"] = {"count": count, "keep": keep}
    want, weights = ps.choose(torch.softmax(total[:, :E], dim=-1), router)
    if renormalize:
        weights = weights / weights.sum(-1, keepdim=True)
    assert torch.equal(chosen.cpu().long(), want) and rel_err(share, weights) < 2e-6
    assert rel_err(gate, torch.sigmoid(total[:, E])) < 1e-6


@pytest.mark.parametrize("shape", [(5, 64, 6, 3, 24, (3, 2), 40), (300, 96, 40, 5, 16, (5, 2), 0), (33, 32, 4, 2, 32, (2, 1), 16),
                                   (2, 48, 4, 1, 20, None, 0), (700, 64, 8, 4, 40, (4, 3), 24), (1, 64, 1, 1, 8, None, 8),
                                   (90, 36, 5, 5, 12, None, 12)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_limited_experts_in_groups_with_a_gated_shared_expert(shape, dtype):
    from test_parts_gpu import Bench
    from flambeau_b200.parts.moe import RoutedExperts
    from flambeau_b200.parts.spec import PartSpec
    n, D, E, K, ff, groups, shared = shape
    dt = DT[dtype]
    b = Bench(dtype, max_step_tokens=1024, cache_tokens=2048)
    shared_spec = PartSpec("feed_forward", "gated_mlp", dict(width=D, inner=shared, activation="limited", limit=0.6, slope=1.702,
                                                             names=("gate", "up", "down")), "m.shared.") if shared else None
    count, keep = groups or (1, 0)
    part = RoutedExperts(b.rt, "m.", width=D, inner=ff, experts=E, top=K, activation="limited", limit=0.9, slope=1.702,
                         gated=True, rule="softmax_of_all", renormalize=False, groups=count, keep_groups=keep,
                         router_bias=False, shared=shared_spec, shared_gate=bool(shared))
    g = torch.Generator().manual_seed(n)
    w = {name: (torch.randn(ts.shape, generator=g) * (0.3 if name.endswith("router") else 0.2)).to(dt)
         for name, ts in part.tensor_specs().items()}
    part.bind({k: v.to(DEV) for k, v in w.items()})
    h = torch.randn(n, D, generator=g).to(dt)
    mlp = {"router": {"experts": E, "top": K}, "expert": {"limit": 0.9}, "shared": {"limit": 0.6} if shared else None}
    if groups:
        mlp["router"]["groups"] = {"count": count, "keep": keep}
    want = ps.routed_ff(h.double(), {k: v.double() for k, v in w.items()}, "m.", mlp)
    for to_stream in (False, True):       # left for the next norm to add, or added to the block's stream by the part
        ctx, x = b.begin([("a" if to_stream else "b", [1] * n, [])], D)
        x.zero_()
        ctx.pending_slabs, ctx.stream_x = 1, x if to_stream else None
        part.forward(ctx, h.to(DEV), ctx.delta)
        b.end()
        assert ctx.pending_slabs == (0 if to_stream else 1) and (ctx.stream_x is x) == to_stream
        out = x if to_stream else ctx.delta_slabs[:ctx.pending_slabs].sum(0)
        # a token whose choice was close may go to another expert in bfloat16: all but a few rows must agree
        err = (out.double().cpu() - want).abs().max(dim=1).values / want.abs().max()
        tol = 2e-5 if dtype == "float32" else 2e-2
        assert int((err > tol).sum()) <= (0 if dtype == "float32" or K == E else n // 50), float(err.max())


GEOMETRIES = [(8, 2, 64, 64, 120, 16), (4, 2, 16, 24, 9, 16), (6, 1, 64, 64, 70, 16), (2, 2, 128, 128, 40, 32), (8, 4, 32, 32, 33, 8),
              (3, 3, 24, 8, 20, 16), (2, 1, 8, 8, 1, 16), (4, 4, 96, 96, 100, 64), (2, 1, 40, 40, 0, 16), (20, 1, 64, 64, 50, 16),
              (2, 1, 256, 256, 64, 16)]


@pytest.mark.parametrize("geometry", GEOMETRIES, ids=lambda g: "h%d-g%d-d%d-e%d-w%d-p%d" % g)
@pytest.mark.parametrize("cap", [0.0, 3.0, 50.0, 1000.0])
@pytest.mark.parametrize("gated", [False, True], ids=["plain", "head-gate"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_with_capped_scores_and_a_gate_per_head(geometry, cap, gated, dtype):
    """Over the paged cache, pages the window has passed given back and unreadable: first tokens, positions around the
    window's length, decoded tokens far into a request and at page borders, portions in mid-page and of two tokens.  The
    key at the window's far edge stands out along the query of head 0, the one just outside it more so.  A cap of 3
    bends most scores of the standing-out keys, one of 50 hardly any; one of 1,000 takes the kernels' other form of the cap."""
    from flambeau_b200.kernels import ops
    nh, nkv, d, e, window, page = geometry
    dt = DT[dtype]
    seqs = [(0, 1), (0, 37), (window, 1), (window + 1, 1), (199, 1), (page * 3 - 1, 1), (page * 3, 1), (page * 2 + 5, 29), (150, 2),
            (63, 70), (10, 300), (window + 40, 1)]
    g = torch.Generator().manual_seed(5)
    scale = 0.9 / math.sqrt(d)
    group = torch.arange(nh) // (nh // nkv)
    qs, ks, vs = [], [], []
    for ctx, n in seqs:
        T = ctx + n
        q, k, v = (torch.randn(m, heads, size, generator=g).to(dt).double() for m, heads, size in
                   ((n, nh, d), (T, nkv, d), (T, nkv, e)))
        for row in {0, n - 1}:
            p = ctx + row
            unit = q[row, 0] / (q[row, 0] ** 2).sum()
            for at, strength in ((p - window + 1, 12.0), (p - window, 30.0)):
                if window and 0 <= at <= p:
                    k[at, 0] = (unit * strength / scale).to(dt).double()
        qs.append(q)
        ks.append(k)
        vs.append(v)
    cache = paged_keys_and_values(seqs, ks, vs, page_size=page, dtype=dt, window=window, given_back=True)
    rows = sum(n for _, n in seqs)
    gates = torch.randn(2, rows, nh + 5, generator=g)
    want = torch.cat([ps_attend(q, k[:, group], v[:, group], scale, cap, window, ctx) for (ctx, n), q, k, v in zip(seqs, qs, ks, vs)])
    if gated:
        want = want * torch.sigmoid(gates.double().sum(0)[:, 3:3 + nh])[:, :, None]
    lens = [n for _, n in seqs]
    multi = [s for s, n in enumerate(lens) if n > 1]
    q_d = torch.cat([q.reshape(q.shape[0], -1) for q in qs]).to(dt).to(DEV).contiguous()
    out = torch.empty((rows, nh * e), dtype=dt, device=DEV)
    rt = SimpleNamespace(status=torch.zeros(1, dtype=torch.int32, device=DEV))
    batch = SimpleNamespace(n_seqs=len(seqs), seq_q_len=lens, seq_q_start_d=i32([sum(lens[:i]) for i in range(len(lens))]),
                            seq_q_len_d=i32(lens), seq_pos_start_d=i32([c for c, _ in seqs]), max_q_len=max(lens),
                            max_kv_len=max(c + n for c, n in seqs), multi_seqs_d=i32(multi), n_multi=len(multi),
                            positions=i32([p for c, n in seqs for p in range(c, c + n)]),
                            row_seq=i32([s for s, n in enumerate(lens) for _ in range(n)]))
    gd = gates.to(DEV)
    ops.paged_attention(SimpleNamespace(batch=batch, runtime=rt), q_d, out, cache, nh, nkv, d, window, scale, vd=e, softcap=cap,
                        head_gate=(gd[0][:, 3:3 + nh], 2, gd.stride(0)) if gated else None, weights_float32=True)
    assert int(rt.status.item()) == 0
    assert rel_err(out, want.reshape(rows, -1)) < (2e-5 if dtype == "float32" else 1.5e-2)


def ps_attend(q, k, v, scale, cap, window, ctx):
    """The oracle's scores, cap, mask and softmax for queries that stand at ctx, ctx + 1, ... of a sequence."""
    s = ps.capped(torch.einsum("ihd,jhd->hij", q, k) * scale, cap or None)
    seen = ps.visible(k.shape[0], window or None)[ctx:]
    return torch.einsum("hij,jhe->ihe", torch.softmax(s.masked_fill(~seen[None], -math.inf), dim=-1), v)


def test_scores_over_the_whole_range_of_a_cap():
    """The bfloat16 kernels' capped scores against the exact function, from scores far below the cap to far above it: one
    query and two keys, so that the output is the softmax of two scores and any error of the cap shows in it."""
    from flambeau_b200.kernels import ops
    d, nh = 64, 1
    targets = [0.0, 1e-3, 0.1, 0.5, 0.9, 1.0, 1.3, 2.0, 4.0, 8.0, 40.0, 200.0]
    cap = 5.0
    for sign in (1.0, -1.0):
        ks = [torch.zeros(2, 1, d) for _ in targets]
        vs = [torch.zeros(2, 1, d) for _ in targets]
        for k, v, t in zip(ks, vs, targets):
            k[0, 0, 0] = torch.tensor(sign * t).bfloat16().float()
            v[0, 0, 0], v[1, 0, 1] = 1.0, 1.0
        seqs = [(1, 1)] * len(targets)
        cache = paged_keys_and_values(seqs, ks, vs, page_size=16, dtype=torch.bfloat16)
        q = torch.zeros(len(targets), d)
        q[:, 0] = 1.0
        out = torch.empty(len(targets), d, dtype=torch.bfloat16, device=DEV)
        rt = SimpleNamespace(status=torch.zeros(1, dtype=torch.int32, device=DEV))
        n = len(targets)
        batch = SimpleNamespace(n_seqs=n, seq_q_len=[1] * n, seq_q_start_d=i32(list(range(n))), seq_q_len_d=i32([1] * n),
                                seq_pos_start_d=i32([1] * n), max_q_len=1, max_kv_len=2, multi_seqs_d=i32([0]), n_multi=0,
                                positions=i32([1] * n), row_seq=i32(list(range(n))))
        ops.paged_attention(SimpleNamespace(batch=batch, runtime=rt), q.bfloat16().to(DEV), out, cache, nh, 1, d, 0, 1.0,
                            softcap=cap, weights_float32=True)
        for i, k in enumerate(ks):
            s = cap * math.tanh(float(k[0, 0, 0]) / cap)
            assert abs(float(out[i, 0]) - 1.0 / (1.0 + math.exp(-s))) < 3e-3, (sign, targets[i])


# ---------------------------------------------------------------------------------------------------------------
# parts alone, through the step context and cache the engine uses
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("sizes", [(4, 2, 32, 20, st.rotation(1e3, 16, 3.0)), (20, 1, 64, 70, st.rotation(1e4, 64, 8.0, 32, 4.0, 0.5)),
                                   (5, 5, 8, 12, st.rotation(100.0, 6, 2.0)), (3, 3, 24, 0, st.rotation(1e4, 24)), (2, 1, 16, 1, None),
                                   (6, 3, 18, 40, st.rotation(500.0, 10, 2.0)), (2, 1, 160, 30, st.rotation(1e4, 64, 2.0)),
                                   (2, 2, 10, 25, st.rotation(1e3, 10, 2.0))],
                         ids=lambda s: "h%d-g%d-d%d-w%d" % s[:4])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_part_whose_values_are_its_keys(sizes, dtype):
    """Norm per head, stretched rotation on part of a head, values as the keys were projected, one gate per head, under
    a window, over steps of portions, single tokens and two tokens against whole sequences.  Weights of the norms far
    from one, so that values taken behind the norm would show."""
    from test_parts_gpu import Bench, bind_random
    from flambeau_b200.cache.manager import CallPlan
    from flambeau_b200.models.saropel import ATTENTION_NAMES
    from flambeau_b200.parts.attention import PagedAttention
    from flambeau_b200.parts.spec import PartSpec
    H, G, d, W, rot = sizes
    width, scale, eps = 48, 0.25, 1e-5
    pos = PartSpec("position", "rotary_half", dict(head_dim=d, theta=rot["base"], rotary_dim=rot["dims"],
                                                   stretch=rot.get("scaling"))) if rot else None
    kw = dict(width=width, num_heads=H, num_kv_heads=G, head_dim=d, window=W, scale=scale, gate="head", values_from_keys=True,
              names=ATTENTION_NAMES, weights_float32=True, position=pos, init_std=0.3 if dtype == "float32" else 0.15,
              qk_norm=PartSpec("norm", "rmsnorm", dict(width=d, eps=eps, init=("one_plus_normal", 0.6))))
    b = Bench(dtype, plans=[CallPlan(kv=PagedAttention(None, "m.", **kw).cache_requirement())])
    part = PagedAttention(b.rt, "m.", **kw)
    Wt = bind_random(part, DT[dtype])
    assert "m.v" not in Wt and Wt["m.g"].shape == (H, width)
    g = torch.Generator().manual_seed(3)
    Hs = {"a": torch.randn(174, width, generator=g).to(DT[dtype]), "b": torch.randn(24, width, generator=g).to(DT[dtype])}
    got = run_mixer_in_steps(b, part, Hs, STEPS, width)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": scale, "rot": rot}
    if W:
        m["mask"] = {"size": W}
    for rid, h in Hs.items():
        want = ps.shared_kv_attention(h.double(), Wt, "m.", m, eps, range(len(h)))
        assert rel_err(got[rid], want) < (2e-5 if dtype == "float32" else 2e-2), rid


@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 9, 1.5), (6, 1, 64, 64, 70, 3.0), (3, 3, 24, 8, 0, 10.0), (2, 1, 128, 128, 1, 2.0),
                                   (3, 1, 20, 20, 33, 1.0)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_part_with_capped_scores(sizes, dtype):
    from test_parts_gpu import Bench, bind_random
    from flambeau_b200.cache.manager import CallPlan
    from flambeau_b200.models.saropel import ATTENTION_NAMES
    from flambeau_b200.parts.attention import PagedAttention
    H, G, d, e, W, cap = sizes
    width, scale = 48, 0.3
    kw = dict(width=width, num_heads=H, num_kv_heads=G, head_dim=d, value_dim=e, window=W, scale=scale, softcap=cap,
              names=ATTENTION_NAMES, weights_float32=True, init_std=0.3 if dtype == "float32" else 0.15)
    b = Bench(dtype, plans=[CallPlan(kv=PagedAttention(None, "m.", **kw).cache_requirement())])
    part = PagedAttention(b.rt, "m.", **kw)
    Wt = bind_random(part, DT[dtype])
    g = torch.Generator().manual_seed(3)
    Hs = {"a": torch.randn(174, width, generator=g).to(DT[dtype]), "b": torch.randn(24, width, generator=g).to(DT[dtype])}
    got = run_mixer_in_steps(b, part, Hs, STEPS, width)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "scale": scale, "softcap": cap}
    if W:
        m["mask"] = {"size": W}
    for rid, h in Hs.items():
        want = ps.capped_attention(h.double(), Wt, "m.", m)
        assert rel_err(got[rid], want) < (2e-5 if dtype == "float32" else 2e-2), rid


@pytest.mark.parametrize("n,width", [(1, 64), (5, 96), (64, 256), (65, 256), (300, 256), (400, 50)])
@pytest.mark.parametrize("ff", [None, "dense", "moe"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_parallel_layer_with_token_input(n, width, ff, dtype):
    """One layer through the engine at sizes where its last products leave shares, one share each, or add to the stream
    themselves: logits of a one-layer model against the plain layer."""
    mlp = {None: None, "dense": st.dense(512), "moe": st.moe(4, 2, 64, 1.0, (2, 1), (48, 0.7))}[ff]
    cfg = {"architecture": "Saropel", "norm": {"eps": 1e-5}, "vocab": 100, "width": width, "token_side": {"dim": 20},
           "embedding": st.bigram(31, 3, 7), "layers": [dict(st.shared_kv(4, 2, 32, 50, st.rotation(1e3, 16, 2.0)), mlp=mlp)]}
    import tempfile
    with tempfile.TemporaryDirectory() as tmp:
        c = make_case(f"layer {n}x{width}", cfg, tmp + "/m", dtype, [n], seed=n)
        run(c, tiny.schedule_whole(c["requests"]), tmp + "/o")


# ---------------------------------------------------------------------------------------------------------------
# whole models under schedules
# ---------------------------------------------------------------------------------------------------------------
SHARP = {"float32": 0.25, "bfloat16": 0.12}
LENGTHS = {"SA": [1, 9, 40, 75, 33, 21, 64, 110], "SB": [2, 70, 17, 48, 150, 5], "SC": [30, 3]}


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
    st.make_folder(folder, cfg, seed=seed, dtype=dtype, sharp=SHARP[dtype], steady_router=dtype == "bfloat16")
    requests = tiny.random_requests({"vocab_size": cfg["vocab"]}, lengths, seed=request_seed)
    pcfg, W = ps.read_folder(folder)
    want = {rid: ps.forward(pcfg, W, toks) for rid, toks in requests.items()}
    return dict(name=name, dtype=dtype, cfg=cfg, folder=folder, requests=requests, want=want,
                tol=tolerance(dtype, pcfg, W, requests))


@pytest.fixture(scope="module", params=[(c, d) for c in ("SA", "SB") for d in ("float32", "bfloat16")],
                ids=lambda p: f"{p[0]}-{p[1]}")
def case(request, tmp_path_factory):
    name, dtype = request.param
    return make_case(name, st.CONFIGS[name], tmp_path_factory.mktemp(f"s{name}{dtype}"), dtype, LENGTHS[name],
                     seed=17 if name == "SA" else 29)


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


def test_last_tokens_one_by_one_past_the_windows(case, tmp_path):
    """The tail is longer than most of the windows, so they pass over decoded tokens and give pages back."""
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
    """A trace as a careless client writes it (tiny.schedule_wild): a slot's kept token must not reach the next request
    that gets the slot."""
    for seed in (3, 4):
        requests, sched = tiny.schedule_wild({"vocab_size": case["cfg"]["vocab"]}, seed=seed)
        pcfg, W = ps.read_folder(case["folder"])
        from flambeau_b200.engine.step import Engine, EngineOptions
        from flambeau_b200.engine.trace import replay
        engine = Engine.from_folder(case["folder"], EngineOptions(dtype=case["dtype"], cache_tokens=1024, max_requests=4,
                                                                  max_step_tokens=512))
        replay(engine, sched.lines(), tmp_path / str(seed))
        got = tiny.read_rows(tmp_path / str(seed), sched, case["cfg"]["vocab"])
        full = {u: ps.forward(pcfg, W, toks).numpy() for u, toks in requests.items() if any(k[0] == u for k in got)}
        for (u, p), row in got.items():
            err = abs(row - full[u][p]).max() / abs(full[u]).max()
            assert err <= case["tol"][0], (seed, u, p, err)


def test_no_token_input_and_an_odd_width(tmp_path):
    for dtype in ("float32", "bfloat16"):
        c = make_case("SC", st.CONFIGS["SC"], tmp_path / dtype, dtype, LENGTHS["SC"], seed=3, request_seed=2)
        run(c, tiny.schedule_portions(c["requests"], sizes=(5, 2, 9)), tmp_path / dtype / "o")
        run(c, tiny.schedule_tail(c["requests"], 12), tmp_path / dtype / "t")


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: widths that are and are not multiples of 8, odd head sizes, windows from one
    key to beyond the requests, caps, stretched and plain rotations, groups of experts, with and without a shared expert,
    a pair table and token input, loops, layers without feed-forward."""
    import random
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(1, 4)):
        mlp = None
        roll = rng.random()
        if roll < 0.35:
            mlp = st.dense(rng.choice([24, 40, 100]))
        elif roll < 0.85:
            count, per = rng.choice([(1, 5), (2, 3), (3, 4), (4, 2), (5, 1)])
            keep = rng.randint(1, count)
            mlp = st.moe(count * per, rng.randint(1, min(keep * per, 4)), rng.choice([8, 16, 24, 40]), rng.uniform(0.5, 2.0),
                         rng.choice([(count, keep), (count, keep), None]), rng.choice([None, (8, 0.7), (32, 1.5)]))
        heads, kv = rng.choice([(1, 1), (2, 1), (4, 2), (6, 3), (3, 3), (18, 1)])
        d = rng.choice([6, 8, 16, 24, 32, 64])
        window = rng.choice([0, 1, 2, 5, 16, 17, 31, 64, 500])
        if rng.random() < 0.5:
            mix = st.capped(heads, kv, d, rng.choice([d, d, 8, 24]), window, rng.uniform(0.5, 8.0), rng.uniform(0.1, 0.4))
        else:
            rot = rng.choice([None, st.rotation(rng.choice([100.0, 1e4, 5e5]), rng.choice([2, d]), rng.choice([None, 2.0, 5.0]),
                                                rng.choice([16, 100, 4096]), rng.choice([32.0, 3.0]), rng.choice([1.0, 0.2]))])
            mix = st.shared_kv(heads, kv, d, window, rot, rng.uniform(0.1, 0.4))
        layers.append(dict(mix, mlp=mlp))
    cfg = {"architecture": "Saropel", "norm": {"eps": rng.choice([1e-5, 1e-6])}, "vocab": rng.randint(50, 400),
           "width": rng.choice([40, 72, 100, 128, 36]), "layers": layers}
    if rng.random() < 0.7:
        cfg["embedding"] = st.bigram(rng.choice([1, 7, 100, 1009]), rng.randint(1, 10 ** 6), rng.randint(1, 10 ** 6))
    if rng.random() < 0.7:
        cfg["token_side"] = {"dim": rng.choice([1, 8, 10, 24])}
    if rng.random() < 0.6:
        start = rng.randint(0, len(layers) - 1)
        cfg["loop"] = {"start": start, "stop": rng.randint(start, len(layers)), "times": rng.randint(1, 3)}
    return cfg


@pytest.mark.parametrize("seed", [401, 402, 403, 404, 405, 406, 407, 408, 409, 410])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configurations_under_a_mixed_schedule(tmp_path, seed, dtype):
    cfg = random_config(seed)
    c = make_case(f"random {seed}", cfg, tmp_path / "m", dtype, [1, 37, 80, 2, 55, 21], seed=seed, request_seed=seed)
    run(c, tiny.schedule_mixed(c["requests"], seed=seed), tmp_path / "o")


def logits_at_the_end(folder, tokens, cut, dtype="float32"):
    """The last position's logits, the request fed as tokens[:cut] and then the rest (a single token when cut is
    len - 1: the position is then a decoded one)."""
    from flambeau_b200.engine.step import Engine, EngineOptions
    engine = Engine.from_folder(folder, EngineOptions(dtype=dtype, cache_tokens=1024, max_requests=2, max_step_tokens=512))
    if cut:
        engine.step([("a", tokens[:cut], [])])
    return engine.step([("a", tokens[cut:], [len(tokens) - cut - 1])], end=["a"])[0].double().cpu()


@pytest.mark.parametrize("window", [1, 2, 11, 16, 17, 64, 70])
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_windows_end_where_they_should_in_prompts_and_in_decoding(tmp_path, window, kind):
    """One layer without feed-forward and without pairs, float32: a token then reaches later positions through its key
    and value alone.  Changing the token just outside the last query's window leaves its logits as they were; changing
    the one just inside moves them.  The last position is once part of a portion, once a decoded token."""
    mix = st.capped(3, 1, 16, 24, window, 4.0) if kind == "attention" else st.shared_kv(3, 1, 16, window, st.rotation(1e4, 8, 2.0))
    cfg = {"architecture": "Saropel", "norm": {"eps": 1e-5}, "vocab": 150, "width": 48, "token_side": {"dim": 8},
           "layers": [dict(mix, mlp=None)]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=8, dtype="float32", sharp=0.12)
    base = tiny.random_requests({"vocab_size": cfg["vocab"]}, [160], seed=1)["r0"]
    p = len(base) - 1

    def moves(at, cut, ref):
        t = list(base)
        t[at] = (t[at] + 1) % cfg["vocab"]
        return float((logits_at_the_end(folder, t, cut) - ref).abs().max()) / float(ref.abs().max())
    for cut in (60, p - 1, p):                      # (p: the last token is decoded alone)
        ref = logits_at_the_end(folder, base, cut)
        assert moves(p - window, cut, ref) < 1e-6, cut
        if window > 1:
            assert moves(p - window + 1, cut, ref) > 1e-5, cut
    pcfg, W = ps.read_folder(folder)
    assert rel_err(logits_at_the_end(folder, base, 37), ps.forward(pcfg, W, base)[-1]) < 1e-4


def test_the_token_before_is_kept_from_step_to_step(tmp_path):
    """A window of one key and no loop: the token before reaches a position through the pair table alone.  It moves the
    logits however the request is cut, the one before it does not; a first token takes the row of its own whatever
    the slot held; a snapshot that comes back into another slot goes on with its own token."""
    from flambeau_b200.engine.step import Engine, EngineOptions
    cfg = {"architecture": "Saropel", "norm": {"eps": 1e-5}, "vocab": 60, "width": 32, "embedding": st.bigram(1009, 31, 7),
           "layers": [dict(st.capped(2, 1, 16, 16, 1, 4.0), mlp=None)]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=4, dtype="float32")
    pcfg, W = ps.read_folder(folder)
    base = [5, 9, 11, 3, 40, 22]
    want = ps.forward(pcfg, W, base)
    for cut in range(len(base)):
        assert rel_err(logits_at_the_end(folder, base, cut), want[-1]) < 1e-4, cut
    other = base[:4] + [41, 22]
    assert rel_err(logits_at_the_end(folder, other, 5), want[-1]) > 1e-2
    assert rel_err(logits_at_the_end(folder, base[:3] + [8, 40, 22], 5), want[-1]) < 1e-4
    engine = Engine.from_folder(folder, EngineOptions(dtype="float32", cache_tokens=512, max_requests=2, max_step_tokens=64))
    for rid in ("a", "b", "c", "d"):                # slots used again
        first = engine.step([(rid, [22], [0])])[0].double().cpu()
        assert rel_err(first, ps.forward(pcfg, W, [22])[0]) < 1e-4, rid
        engine.step([(rid, [7, 8], [])], end=[rid])
    engine.step([("x", base[:5], [])])
    kept = engine.snapshot("x")
    engine.finish("x")
    engine.step([("y", [1, 2, 3], []), ("z", [4], [])], end=["y"])
    engine.restore("x", kept)
    assert rel_err(engine.step([("x", base[5:], [0])])[0].double().cpu(), want[-1]) < 1e-4


def test_a_far_key_among_hundreds_is_found(tmp_path):
    """Attention whose values are its keys, no mask, float32: one head's maps are rebuilt so that its query for one token
    points along another token's key (unrotated dimensions only).  Where the first stands last and the second hundreds of
    positions back and nowhere else, that far key takes most of the head's softmax, so that losing the key, or its page,
    would move the logits by far more than any rounding."""
    cfg = {"architecture": "Saropel", "norm": {"eps": 1e-5}, "vocab": 90, "width": 32,
           "layers": [dict(st.shared_kv(2, 1, 16, 0, st.rotation(1e4, 4, 2.0), 1.0), mlp=None)]}
    folder = st.make_folder(tmp_path / "m", cfg, seed=10, dtype="float32", sharp=0.3)
    pcfg, W = ps.read_folder(folder)
    asks, answers = 85, 84
    h = ps.norm_around_one(W["embed"][[asks, answers]], W["l0.norm1"], 1e-5)
    tensors = st.read_tensors(folder)
    tensors["l0.mix.q.norm"][:] = 1.5
    tensors["l0.mix.k.norm"][:] = 1.0
    tensors["l0.mix.k"][8] = (8.0 * h[1] / (h[1] ** 2).sum()).float()        # the answer's key stands out in dimension 8
    tensors["l0.mix.q"][:16] = 0.0
    tensors["l0.mix.q"][8] = (8.0 * h[0] / (h[0] ** 2).sum()).float()
    st.write_tensors(folder, tensors)
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


def test_a_table_that_all_layers_read_is_on_the_device_once(tmp_path):
    from flambeau_b200.config.saropel import SaropelConfig
    from flambeau_b200.engine.step import Engine, EngineOptions
    folder = st.make_folder(tmp_path / "m", st.CONFIG_SA, seed=2, dtype="bfloat16")
    opts = dict(dtype="bfloat16", cache_tokens=256, max_requests=2, max_step_tokens=64)
    for engine in (Engine.from_folder(folder, EngineOptions(**opts)),
                   Engine.from_config(SaropelConfig.from_dict(st.CONFIG_SA), options=EngineOptions(**opts))):
        assert len({layer.table.data_ptr() for layer in engine.model.layers}) == 1


# ---------------------------------------------------------------------------------------------------------------
# generation through the entry point and the scheduler
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name,dtype", [("SA", "float32"), ("SB", "bfloat16"), ("SA", "bfloat16")])
def test_greedy_generation(tmp_path, name, dtype):
    from flambeau_b200 import generate
    cfg = st.CONFIGS[name]
    folder = st.make_folder(tmp_path / "m", cfg, seed=41, dtype=dtype, sharp=SHARP[dtype], steady_router=dtype == "bfloat16")
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
    cfg = st.CONFIGS["SC"]
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
