"""Saropel beside Tubepel at equal size: prefill and decode throughput and, kernel by kernel, how far each is from its
roofline.

`bench.py --only saropel` runs, for each size of SIZES, a Saropel model (parallel blocks: attention whose values are
its keys in front of routed experts chosen within groups, and capped attention in front of a dense gated feed-forward,
in turn; an embedding of token pairs and a token input behind every layer) and a Tubepel model (the framework's closest
design, here on a plain residual stream with windowed grouped attention in every layer: a sink, an output gate, routed
gated experts and a dense squared-ReLU feed-forward in turn) with the same width, heads, head size, window, vocabulary,
experts and number of layers, both with random weights in bfloat16, through the same engine calls: one decode step of
`batch` sequences that each hold `context` tokens, and one step of `prefill` prompt tokens.  Per design it reports
tokens a second and, per launcher (CUDA events around every launcher call of an eager step, so serialised kernels),
launches and microseconds a launch, the work of one launch and the fraction of the measured peak that bounds it.
`like` pairs every kernel of the new design with the kernel of Tubepel that does the like job and gives the ratio of
their fractions (below 0.5: more than twice as far from the roofline).

Work of one launch over `rows` rows (D = width, C = columns of a layer's token input):
  attention        4 * seen * heads * head size flops; bytes: live keys and values of the key/value heads + queries and
                   outputs
  cache_write      the projection's float32 rows in, the rounded queries and the cache rows out (where the values are
                   the keys, one row in and two out)
  norm             the stream in and out, the pending output in (float32), normalised rows out; where the products have
                   added to the stream themselves, the stream in and the rows out
  settle           the stream in, its rows in 16 bits out; for few rows also the pending output in and the stream out
  token_gate       the gate's float32 rows in, the token's columns in, C columns out
  pair_embedding   two table rows in, one float32 row out
  routed_product   6 * pairs * D * expert inner size flops for both products; bytes: the weights of the experts that
                   were chosen, once
  expert_gather    the tokens' rows in (once per chosen expert) and out
  expert_combine   the chosen experts' rows and the shared expert's in, the stream in and out
"""
from __future__ import annotations

import gc

import torch

from ..config.saropel import SaropelConfig
from ..config.tubepel import TubepelConfig
from ..engine.batch import Entry
from ..engine.step import Engine, EngineOptions
from ..kernels import ops
from . import work, workloads
from .compare import PAGE
from .compare_tubepel import CLASS_OF as TUBEPEL_CLASSES, SIZES as TUBEPEL_SIZES
from .timers import SectionTimer

# what Saropel adds to the sizes of measure/compare_tubepel.py: groups of experts and how many of them are kept, columns
# of a layer's token input, buckets of the pair table, the cap
SIZES = {k: dict(v, groups=4, keep=2, side=256, buckets=65521, softcap=30.0) for k, v in TUBEPEL_SIZES.items()}

CLASS_OF = dict(TUBEPEL_CLASSES, rope_kv_write="cache_write", qk_norm_rope_kv_write="cache_write_normed",
                norm_add_rms_norm="norm", add_slabs="settle", embedding_pairs="pair_embedding", embedding="embedding",
                sigmoid_gate="output_gate")

# (kernel of Saropel, the like kernel of Tubepel); kernels that only Saropel has are set beside the kernel of Tubepel
# that is bound by the same thing (rows through memory)
LIKE = [("attention_capped", "attention"), ("attention_head_gate", "attention"), ("cache_write", "cache_write"),
        ("cache_write_normed", "cache_write"), ("norm", "norm"), ("settle", "norm"), ("token_gate", "output_gate"),
        ("pair_embedding", "embedding"), ("routed_product", "routed_product"), ("expert_gather", "expert_gather"),
        ("expert_combine", "expert_combine"), ("router", "router"), ("expert_order", "expert_order"),
        ("gate_mul", "gate_mul")]


def saropel_config(size: dict, layers: int) -> SaropelConfig:
    d = size["qk_row"]
    moe = {"kind": "moe", "expert": {"ff": size["expert_ff"], "limit": 7.0}, "shared": {"ff": size["shared_ff"], "limit": 7.0},
           "router": {"experts": size["experts"], "top": size["top"], "groups": {"count": size["groups"], "keep": size["keep"]}}}
    sizes = {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": d, "vdim": d, "mask": {"size": size["window"]},
             "scale": d ** -0.5}
    shared = {"type": "attention_2", "mlp": moe, "mixer": dict(sizes, rot={
        "base": 1e6, "dims": d // 2, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}})}
    capped = {"type": "attention", "mlp": {"kind": "dense", "ff": size["dense_ff"]}, "mixer": dict(sizes, softcap=size["softcap"])}
    return SaropelConfig.from_dict({
        "architecture": "Saropel", "norm": {"eps": 1e-6}, "vocab": size["vocab"], "width": size["width"],
        "token_side": {"dim": size["side"]},
        "embedding": {"bigram": {"buckets": size["buckets"], "mul_prev": 31, "mul_cur": 17}},
        "layers": [capped if i % 2 == 0 else shared for i in range(layers)]})


def tubepel_config(size: dict, layers: int) -> TubepelConfig:
    moe = {"kind": "moe", "router": {"experts": size["experts"], "top": size["top"]}, "expert": {"ff": size["expert_ff"]},
           "shared": {"ff": size["shared_ff"]}}
    mixer = {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": size["qk_row"], "vdim": size["qk_row"],
             "mask": {"size": size["window"]}, "rot": {"base": 1e6, "dims": size["qk_row"] // 2}, "scale": size["qk_row"] ** -0.5}
    return TubepelConfig.from_dict({
        "architecture": "Tubepel", "norm": {"eps": 1e-6}, "vocab": size["vocab"], "width": size["width"],
        "layers": [{"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": size["dense_ff"]} if i % 2 == 0 else moe}
                   for i in range(layers)]})


def configs(size: dict, layers: int) -> dict:
    return {"saropel": saropel_config(size, layers), "tubepel": tubepel_config(size, layers)}


def sections_by_class(engine, entries, end=(), reps: int = 3) -> dict:
    """class -> (launches, milliseconds) per step of one eager step; attention launches are told apart by what their
    scores and outputs pass, products are keyed by their matrix."""
    was = engine.use_graphs
    engine.use_graphs = False
    try:
        engine.step(entries, end=end)
        totals: dict = {}
        for _ in range(reps):
            torch.cuda._sleep(int(40.0 * 2.0e6))
            with SectionTimer() as t:
                logits = engine.step(entries, end=end)
                if logits is not None:
                    ops.sample(logits, torch.zeros(logits.shape[0], dtype=torch.int32, device=logits.device))
            for what, note, ms in t.sections():
                key = CLASS_OF.get(what) or (f"product {note[1]}x{note[2]}" if what.startswith("gemm") and note else what)
                if key == "attention" and note and note[3]:
                    key += "_" + note[3]
                n, total = totals.get(key, (0, 0.0))
                totals[key] = (n + 1, total + ms)
        return {k: (n / reps, total / reps) for k, (n, total) in totals.items()}
    finally:
        engine.use_graphs = was


def kernel_work(design: str, size: dict, rows: int, contexts) -> dict:
    """class -> flops / bytes of one launch."""
    D, W, H, G, d = size["width"], size["window"], size["heads"], size["kv_heads"], size["qk_row"]
    pairs = rows * size["top"]
    experts_read = min(size["experts"], pairs)
    decoding = len(contexts) == rows
    if decoding:
        seen = keys = sum(work.live_keys(c, W) for c in contexts)
    else:
        ctx = contexts[0]
        seen, keys = work.keys_seen(range(ctx - rows, ctx), W), ctx - max(0, ctx - rows - W + 1)
    attention = dict(flops=4.0 * seen * H * d, bytes=keys * G * 2 * d * 2 + rows * H * 2 * d * 2)
    # Norms.  Few rows: the stream in and out, what is pending in, rows out.  Over a portion the products and the
    # experts' sum have joined the stream (Saropel's norms always take the token input, which passes a norm of its own).
    full, bare = rows * D * (4 + 4 + 4 + 2), rows * D * (4 + 2)
    works = {
        "attention": attention, "attention_capped": attention, "attention_head_gate": attention,
        "cache_write": dict(bytes=rows * (H + 2 * G) * d * (4 + 2)),
        "cache_write_normed": dict(bytes=rows * ((H + G) * d * 4 + (H + 2 * G) * d * 2)),
        "norm": dict(bytes=full if decoding or design == "saropel" else bare),
        "settle": dict(bytes=full if decoding else bare),
        "token_gate": dict(bytes=rows * size["side"] * (4 + 2 + 2)),
        "output_gate": dict(bytes=rows * H * d * (2 + 2 + 4)),
        "pair_embedding": dict(bytes=rows * D * (2 + 2 + 4)), "embedding": dict(bytes=rows * D * (2 + 4)),
        "routed_product": dict(flops=6.0 * pairs * D * size["expert_ff"] / 2.0,
                               bytes=experts_read * 3 * D * size["expert_ff"] * 2 / 2.0),     # (two launches for it)
        "expert_gather": dict(bytes=pairs * D * 2 * 2), "expert_combine": dict(bytes=rows * D * 4 * (size["top"] + 3)),
        "expert_order": dict(bytes=pairs * 4 * 3), "router": dict(bytes=rows * size["experts"] * 4),
        "gate_mul": dict(bytes=rows * size["shared_ff"] * (8 + 2)), "activation": dict(bytes=rows * size["dense_ff"] * (4 + 2)),
    }
    return works


def kernel_table(engine, design: str, size: dict, entries, end, rows: int, contexts, peaks: dict) -> dict:
    secs = sections_by_class(engine, entries, end=end)
    works = kernel_work(design, size, rows, contexts)
    table = {}
    for key, (n, total) in sorted(secs.items()):
        r = {"launches": round(n, 2), "us": round(total * 1e3 / max(n, 1e-9), 2)}
        w = works.get(key)
        if key.startswith("product ") and rows > 0:
            N, K = (int(x) for x in key[8:].split("x"))
            m = rows if K != size["width"] or N != size["vocab"] else (rows if len(contexts) == rows else 1)
            w = dict(flops=2.0 * m * N * K, bytes=N * K * 2 + m * K * 2 + m * N * 4)
        if w and r["us"] > 0:
            sec = r["us"] * 1e-6
            by_mem = w.get("bytes", 0.0) / sec / 1e9 / peaks["hbm_gbs"]
            by_math = w.get("flops", 0.0) / sec / 1e12 / peaks["bf16_tflops"]
            r.update(bound="hbm" if by_mem >= by_math else "tensor", frac=round(max(by_mem, by_math), 4))
        table[key] = r
    return table


def measure(name: str, size: dict, layers: int, batch: int, context: int, prefill: int, steps: int, warmup: int,
            peaks: dict, gen, say) -> dict:
    out = {"size": dict(size), "layers": layers, "batch": batch, "context": context, "prefill_tokens": prefill}
    for design, cfg in configs(size, layers).items():
        say(f"{name}: building {design}, {layers} layers")
        live = min(context, size["window"] + PAGE)
        per_seq = -(-(live + 2 * PAGE + steps + warmup + 64) // PAGE) * PAGE
        engine = Engine.from_config(cfg, seed=0, options=EngineOptions(
            dtype="bfloat16", page_size=PAGE, cache_tokens=max(batch * per_seq + 512, prefill + PAGE),
            max_requests=batch, max_step_tokens=max(prefill, batch), max_seq_len=context + 4096))
        workloads.randomise_cache(engine)
        ms, launches = workloads.decode_device(engine, batch, context, steps, warmup, gen)
        pre_ms = workloads.prefill_step(engine, prefill, gen)
        rec = {"decode_ms": round(ms, 4), "decode_tok_s": round(batch / (ms / 1e3), 1), "launches_per_step": launches,
               "prefill_ms": round(pre_ms, 3), "prefill_tok_s": round(prefill / (pre_ms / 1e3), 1),
               "weight_bytes": engine.model.step_weight_bytes(), "kv_bytes_per_token": engine.cache.kv_bytes_per_token()}
        # what a decode step must read: every weight that takes part (of the routed experts those that the batch's
        # tokens are expected to choose between them, each once) and the live keys and values
        E, K = size["experts"], size["top"]
        distinct = E * (1.0 - (1.0 - K / E) ** batch)
        nbytes = work.decode_step_bytes(rec["weight_bytes"], rec["kv_bytes_per_token"], [context] * batch, size["window"])
        nbytes += layers // 2 * (distinct - K) * 3 * size["width"] * size["expert_ff"] * 2
        rec["decode_bytes"] = int(nbytes)
        rec["decode_hbm_frac"] = round(nbytes / (ms / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
        vocab = engine.model.vocab_size
        ids = workloads.seat(engine, [context] * batch)
        entries = [Entry(r, [int(torch.randint(0, vocab, (1,), generator=gen))], [0]) for r in ids]
        toks = torch.randint(0, vocab, (prefill,), generator=gen).tolist()
        rec[f"decode_b{batch}"] = kernel_table(engine, design, size, entries, (), batch, [context] * batch, peaks)
        engine.cache.release_all()
        rec[f"prefill_{prefill}"] = kernel_table(engine, design, size, [Entry("prompt", toks, [prefill - 1])], ("prompt",),
                                                 prefill, [prefill], peaks)
        engine.cache.release_all()
        out[design] = rec
        engine = None
        gc.collect()
        torch.cuda.empty_cache()
    s, t = out["saropel"], out["tubepel"]
    out["saropel_over_tubepel"] = {"decode_tok_s": round(s["decode_tok_s"] / t["decode_tok_s"], 3),
                                   "prefill_tok_s": round(s["prefill_tok_s"] / t["prefill_tok_s"], 3)}
    like = {}
    for label in (f"decode_b{batch}", f"prefill_{prefill}"):
        rows = {}
        for ours, theirs in LIKE:
            a, b = s[label].get(ours), t[label].get(theirs)
            if a and b and "frac" in a and "frac" in b and b["frac"] > 0:
                rows[ours] = {"like": theirs, "frac": a["frac"], "like_frac": b["frac"], "us": a["us"], "like_us": b["us"],
                              "ratio": round(a["frac"] / b["frac"], 3)}
        like[label] = rows
    out["like"] = like
    return out


def run(sizes, layers: int, batch: int, prefill: int, steps: int, warmup: int, peaks: dict, gen, say) -> dict:
    result = {}
    for name in sizes:
        size = SIZES[name]
        result[name] = measure(name, size, layers, batch, 2 * size["window"], prefill, steps, warmup, peaks, gen, say)
    return result
