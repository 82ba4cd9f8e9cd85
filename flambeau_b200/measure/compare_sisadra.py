"""Sisadra beside the framework's closest designs at equal size: prefill and decode throughput and, kernel by kernel, how
far each is from its roofline.

`bench.py --only sisadra` runs, for each size of SIZES, a Sisadra model (differential attention within chunks, attention
over latents, differential attention, the gated delta rule with a decay per key channel, in turn; plain feed-forwards, none
behind the recurrence; a pair embedding, a cap on the logits) and models of three designs that have a like mechanism each,
with the same width, heads, head sizes, vocabulary and number of layers: Zedivik (differential attention under a window),
Fegizen (attention over latents of the same row size; linear attention with a decay per key channel) and Nodepel (the gated
delta rule with a decay per head; a norm and a rotation on the way to the cache).  All have random weights in bfloat16 and go
through the same engine calls: one decode step of `batch` sequences that each hold `context` tokens, and one step of
`prefill` prompt tokens.  Per design it reports tokens a second and, per launcher (CUDA events around every launcher call
of an eager step, so serialised kernels), launches and microseconds a launch, the work of one launch and the fraction of
the measured peak that bounds it.  `like` pairs every kernel of the new design with the kernel that does the like job and
gives the ratio of their fractions (below 0.5: more than twice as far from the roofline).

Work of one launch over `rows` rows (D = width):
  diff_attention_mma    4 * seen * heads * (key size + value size) flops; bytes: live keys and values + queries and outputs
  paged_attention_mma   over latents: 4 * seen * heads * row flops; bytes: live rows + queries and outputs
  gdr_channel_recurrent per token and head 7 * dk * dv flops (the decay, S^T k and S^T q, the rank-one update), float32 on the
                        CUDA cores (gdr_recurrent 8, its decay entering with the update; gla_recurrent 5); per request the
                        state once in and out, per token its rows
  low_rank_maps         2 * rows * middle * outputs flops; bytes: weights, the middles in, both results out (float32)
  gdr_prepare           the projection's float32 rows in (once), q, k and v out
  qk_norm_rope_kv_write, qkv_bias_cache_write, mla_latents   the projection's float32 rows in, q and the cache rows out
  head_linear           the mean of its two uses: rows in and out, weights; 2 * rows * heads * in * out flops
  norms                 the stream in, normalised rows out (counted as 16-bit); where something joins the stream, a pending
                        output in and the stream out
"""
from __future__ import annotations

import gc

import torch

from ..config.sisadra import SisadraConfig
from ..engine.batch import Entry
from ..engine.step import Engine, EngineOptions
from ..kernels import ops
from . import work, workloads
from .compare import PAGE, configs as zedivik_configs
from .compare_fegizen import SIZES as FEGIZEN_SIZES, fegizen_config
from .compare_nodepel import configs as nodepel_configs, fp32_fma_tflops
from .timers import SectionTimer

# what Sisadra adds to (or sets otherwise than) the sizes of measure/compare_fegizen.py: the size of one score map, the
# feed-forward, the pair table, the cap; equal heads in the recurrence; a narrow middle as wide as a head
SIZES = {
    "1b": dict(FEGIZEN_SIZES["1b"], map_dim=64, ff=8192, buckets=65521, softcap=30.0, r_qk_heads=16),
    "7b": dict(FEGIZEN_SIZES["7b"], map_dim=64, ff=14336, buckets=65521, softcap=30.0, r_qk_heads=32),
}

# (kernel of Sisadra, design, the like kernel there)
LIKE = [("diff_attention_mma", "zedivik", "diff_attention_mma"), ("qk_norm_rope_kv_write", "nodepel", "qk_norm_rope_kv_write"),
        ("paged_attention_mma", "fegizen", "paged_attention_mma"), ("mla_latents", "fegizen", "mla_latents"),
        ("head_linear", "fegizen", "head_linear"), ("gdr_channel_recurrent", "nodepel", "gdr_recurrent"),
        ("gdr_channel_recurrent", "fegizen", "gla_recurrent"), ("gdr_prepare", "nodepel", "gdr_prepare"),
        ("low_rank_maps", "fegizen", "gla_prepare"), ("gdr_out_norm", "nodepel", "gdr_out_norm"),
        ("add_layer_norm", "fegizen", "add_layer_norm"), ("activation", "zedivik", "gate_mul"),
        ("embedding_pairs", "zedivik", "embedding"), ("softcap_rows", "zedivik", "embedding")]


def sisadra_config(size: dict, layers: int) -> SisadraConfig:
    d, W = size["map_dim"], size["window"]
    mlp = {"kind": "dense", "ff": size["ff"]}
    attention = {"type": "attention", "mlp": mlp, "mixer": {
        "heads": size["heads"], "kv_heads": size["kv_heads"], "dim": d, "vdim": size["v_row"], "mask": {"size": W},
        "scale": d ** -0.5, "diff": 0.5,
        "rot": {"base": 1e6, "dims": d, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    latent = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": size["heads"], "dim": size["dim"], "vdim": size["vdim"], "kv_rank": size["kv_rank"] + size["rot_dim"],
        "scale": size["dim"] ** -0.5}}
    delta = {"type": "channel_delta", "mlp": None, "mixer": {
        "heads": size["r_heads"], "kv_heads": size["r_qk_heads"], "dim": size["r_dk"], "vdim": size["r_dv"], "conv": size["conv"]}}
    order = [attention, latent, attention, delta]
    return SisadraConfig.from_dict({
        "architecture": "Sisadra", "norm": {"eps": 1e-6}, "vocab": size["vocab"], "width": size["width"],
        "logit_softcap": size["softcap"],
        "embedding": {"scale": 1.0, "bigram": {"buckets": size["buckets"], "mul_prev": 31, "mul_cur": 17}},
        "layers": [order[i % 4] for i in range(layers)]})


def configs(size: dict, layers: int) -> dict:
    return {"sisadra": sisadra_config(size, layers), "zedivik": zedivik_configs(size, layers)["zedivik"],
            "fegizen": fegizen_config(size, layers), "nodepel": nodepel_configs(size, layers)["nodepel"]}


def sections(engine, entries, end=(), reps: int = 3) -> dict:
    """launcher -> (launches, milliseconds, bytes) per step of one eager step; products are keyed by their matrix.  Bytes are
    counted here for the launches whose work depends on what is pending (the norms: the stream in, a pending output in,
    both written back where something joined, 16-bit rows out)."""
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
                key = f"product {note[1]}x{note[2]}" if what.startswith("gemm") and "grouped" not in what and note else what
                n, total, nbytes = totals.get(key, (0, 0.0, 0.0))
                if what == "add_layer_norm":
                    rows, width, pending, bias, all_rows = note
                    nbytes += rows * width * (4 + 2 + 4 * pending + (4 if all_rows and (pending or bias) else 0))
                totals[key] = (n + 1, total + ms, nbytes)
        return {k: (n / reps, total / reps, nbytes / reps) for k, (n, total, nbytes) in totals.items()}
    finally:
        engine.use_graphs = was


def kernel_work(design: str, size: dict, rows: int, contexts, layers: int) -> dict:
    """launcher -> flops / fma_flops / bytes of one launch."""
    D, W, H, G = size["width"], size["window"], size["heads"], size["kv_heads"]
    Hr, dk, dv, V = size["r_heads"], size["r_dk"], size["r_dv"], size["vocab"]
    Gr = size["r_qk_heads"]
    decoding = len(contexts) == rows
    n_seqs = len(contexts) if decoding else 1

    def visible(window, chunk):
        """(query, visible key) pairs, and keys that are read."""
        if decoding:
            live = [min(c, window) if window else c - (c - 1) // chunk * chunk if chunk else c for c in contexts]
            return sum(live), sum(live)
        ctx = contexts[0]
        if chunk:
            return sum(p - p // chunk * chunk + 1 for p in range(ctx - rows, ctx)), ctx - (ctx - rows) // chunk * chunk
        return work.keys_seen(range(ctx - rows, ctx), window), ctx - (max(0, ctx - rows - W + 1) if window else 0)
    row = size["kv_rank"] + size["rot_dim"]
    seen, keys = visible(0, W) if design == "sisadra" else visible(W, 0)
    l_seen, l_keys = visible(0, 0) if design == "sisadra" else visible(W, 0)
    maps = size["qk_row"] // 2
    diff = dict(flops=4.0 * seen * H * (maps + size["v_row"]),
                bytes=keys * G * (size["qk_row"] + size["v_row"]) * 2 + rows * H * (size["qk_row"] + size["v_row"]) * 2)
    cols = H * size["qk_row"] + G * (size["qk_row"] + size["v_row"])
    full, bare = rows * D * (4 + 4 + 4 + 2), rows * D * (4 + 2)
    state = n_seqs * 2 * Hr * dk * dv * 4
    works = {
        "diff_attention_mma": diff, "qk_norm_rope_kv_write": dict(bytes=rows * cols * (4 + 2)),
        "qkv_bias_cache_write": dict(bytes=rows * cols * (4 + 2)),
        "add_rms_norm": dict(bytes=full if decoding else bare), "norm_add_rms_norm": dict(bytes=full),
        "embedding": dict(bytes=rows * D * (2 + 4)), "embedding_pairs": dict(bytes=rows * D * (2 + 2 + 4)),
        "gate_mul": dict(bytes=rows * size["ff"] * (2 * 4 + 2)), "activation": dict(bytes=rows * size["ff"] * (4 + 2)),
        "softcap_rows": dict(bytes=n_seqs * V * 8), "gdr_out_norm": dict(bytes=rows * Hr * dv * (4 + 4 + 2)),
        "gdr_recurrent": dict(fma_flops=8.0 * rows * Hr * dk * dv, bytes=state + rows * 4 * (2 * Gr * dk + 2 * Hr * dv)),
        "gdr_prepare": dict(bytes=rows * 4 * 2 * (2 * Gr * dk + Hr * dv + Hr)),
        "gla_recurrent": dict(fma_flops=5.0 * rows * Hr * dk * dv, bytes=state + rows * 4 * (3 * Hr * dk + 2 * Hr * dv)),
        "gla_prepare": dict(bytes=rows * 4 * (2 * Hr * dk + Hr * dv + 16 + 3 * Hr * dk + Hr * dv)),
    }
    if design == "nodepel":
        works["paged_attention_mma"] = dict(flops=4.0 * seen * H * size["qk_row"],
                                            bytes=keys * G * (size["qk_row"] + size["v_row"]) * 2 + rows * H * 4 * size["qk_row"])
    if design == "sisadra":
        mid = dk                                           # (what the random weights draw)
        works["gdr_channel_recurrent"] = dict(fma_flops=7.0 * rows * Hr * dk * dv,
                                              bytes=state + rows * 4 * (2 * Gr * dk + Hr * dk + 2 * Hr * dv))
        works["low_rank_maps"] = dict(flops=2.0 * rows * mid * Hr * (dk + dv),
                                      bytes=mid * Hr * (dk + dv) * 2 + rows * 4 * (2 * mid + Hr * (dk + dv)))
        works["paged_attention_mma"] = dict(flops=4.0 * l_seen * H * row, bytes=l_keys * row * 2 + 2 * rows * H * row * 2)
        works["mla_latents"] = dict(bytes=rows * row * (4 + 2))
        works["head_linear"] = dict(flops=2.0 * rows * H * row * (size["dim"] + size["vdim"]) / 2.0,
                                    bytes=(rows * H * (size["dim"] * 4 + 2 * row * 2 + size["vdim"] * 2)
                                           + H * row * (size["dim"] + size["vdim"]) * 2) / 2.0)
    if design == "fegizen":
        q = size["q_rank"]
        works["paged_attention_mma"] = dict(flops=4.0 * l_seen * H * row, bytes=l_keys * row * 2 + 2 * rows * H * row * 2)
        works["mla_latents"] = dict(bytes=rows * (q + row) * (4 + 2))
        works["head_linear"] = dict(flops=2.0 * rows * H * size["kv_rank"] * (size["dim"] + size["vdim"]) / 2.0,
                                    bytes=(rows * H * ((size["dim"] + size["rot_dim"]) * 4 + 2 * row * 2 + size["vdim"] * (2 + 4))
                                           + H * size["kv_rank"] * (size["dim"] + size["vdim"]) * 2) / 2.0)
    return works


def kernel_table(engine, design: str, size: dict, entries, end, rows: int, contexts, layers: int, peaks: dict) -> dict:
    secs = sections(engine, entries, end=end)
    works = kernel_work(design, size, rows, contexts, layers)
    fma_peak = fp32_fma_tflops(engine.runtime.device)
    table = {}
    for key, (n, total, nbytes) in sorted(secs.items()):
        r = {"launches": round(n, 2), "us": round(total * 1e3 / max(n, 1e-9), 2)}
        w = dict(bytes=nbytes / n) if nbytes else works.get(key)
        if key.startswith("product "):
            N, K = (int(x) for x in key[8:].split("x"))
            m = len(contexts) if (N, K) == (size["vocab"], size["width"]) else rows
            w = dict(flops=2.0 * m * N * K, bytes=N * K * 2 + m * K * 2 + m * N * 4)
        if w and r["us"] > 0:
            sec = r["us"] * 1e-6
            fracs = {"hbm": w.get("bytes", 0.0) / sec / 1e9 / peaks["hbm_gbs"],
                     "tensor": w.get("flops", 0.0) / sec / 1e12 / peaks["bf16_tflops"],
                     "fp32 fma": w.get("fma_flops", 0.0) / sec / 1e12 / fma_peak}
            bound = max(fracs, key=fracs.get)
            r.update(bound=bound, frac=round(fracs[bound], 4))
        table[key] = r
    return table


def measure(name: str, size: dict, layers: int, batch: int, context: int, prefill: int, steps: int, warmup: int,
            peaks: dict, gen, say) -> dict:
    out = {"size": dict(size), "layers": layers, "batch": batch, "context": context, "prefill_tokens": prefill}
    for design, cfg in configs(size, layers).items():
        say(f"{name}: building {design}, {layers} layers")
        per_seq = -(-(context + 2 * PAGE + steps + warmup + 64) // PAGE) * PAGE
        engine = Engine.from_config(cfg, seed=0, options=EngineOptions(
            dtype="bfloat16", page_size=PAGE, cache_tokens=max(batch * per_seq + 512, prefill + PAGE),
            max_requests=batch, max_step_tokens=max(prefill, batch), max_seq_len=context + 4096))
        workloads.randomise_cache(engine)
        ms, launches = workloads.decode_device(engine, batch, context, steps, warmup, gen)
        pre_ms = workloads.prefill_step(engine, prefill, gen)
        rec = {"decode_ms": round(ms, 4), "decode_tok_s": round(batch / (ms / 1e3), 1), "launches_per_step": launches,
               "prefill_ms": round(pre_ms, 3), "prefill_tok_s": round(prefill / (pre_ms / 1e3), 1),
               "weight_bytes": engine.model.step_weight_bytes(), "kv_bytes_per_token": engine.cache.kv_bytes_per_token(),
               "state_bytes_per_request": engine.cache.state_bytes_per_request()}
        # what a decode step must read: the weights that take part (all of a dense model's), the live keys and values of every
        # group, and the states in and out
        if design in ("sisadra", "zedivik"):
            nbytes = rec["weight_bytes"] + 2 * batch * rec["state_bytes_per_request"]
            for g in engine.cache.groups:
                chunk, window = g.req.chunk, g.req.window
                live = context - (context - 1) // chunk * chunk if chunk else min(context, window) if window else context
                nbytes += batch * live * g.bytes_per_token()
            rec["decode_bytes"] = int(nbytes)
            rec["decode_hbm_frac"] = round(nbytes / (ms / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
        vocab = engine.model.vocab_size
        ids = workloads.seat(engine, [context] * batch)
        entries = [Entry(r, [int(torch.randint(0, vocab, (1,), generator=gen))], [0]) for r in ids]
        toks = torch.randint(0, vocab, (prefill,), generator=gen).tolist()
        rec[f"decode_b{batch}"] = kernel_table(engine, design, size, entries, (), batch, [context] * batch, layers, peaks)
        engine.cache.release_all()
        rec[f"prefill_{prefill}"] = kernel_table(engine, design, size, [Entry("prompt", toks, [prefill - 1])], ("prompt",),
                                                 prefill, [prefill], layers, peaks)
        engine.cache.release_all()
        out[design] = rec
        engine = None
        gc.collect()
        torch.cuda.empty_cache()
    s = out["sisadra"]
    for other in ("zedivik", "fegizen", "nodepel"):
        out[f"sisadra_over_{other}"] = {k: round(s[k] / out[other][k], 3) for k in ("decode_tok_s", "prefill_tok_s")}
    like = {}
    for label in (f"decode_b{batch}", f"prefill_{prefill}"):
        rows = {}
        for ours, design, theirs in LIKE:
            a, b = s[label].get(ours), out[design][label].get(theirs)
            if a and b and "frac" in a and "frac" in b and b["frac"] > 0:
                rows[f"{ours} / {design} {theirs}"] = {"bound": a["bound"], "frac": a["frac"], "like_frac": b["frac"], "us": a["us"],
                                                       "like_us": b["us"], "ratio": round(a["frac"] / b["frac"], 3)}
        like[label] = rows
    out["like"] = like
    return out


def run(sizes, layers: int, batch: int, prefill: int, steps: int, warmup: int, peaks: dict, gen, say) -> dict:
    result = {}
    for name in sizes:
        size = SIZES[name]
        # the timed steps end in front of a chunk's edge: behind it a token would see hardly any keys
        context = 2 * size["window"] - steps - warmup - 16
        result[name] = measure(name, size, layers, batch, context, prefill, steps, warmup, peaks, gen, say)
    return result
