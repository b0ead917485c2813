"""Prefill and decode throughput of the serving models on layers of realistic size with random weights: the Ginisun, Pufevik, Mepupel and Vemepel decoders beside a Llama decoder
of the same width and the same number of feed-forward neurons per token (Pufevik also has its attention sizes; its layers alternate between the two kinds; Mepupel and Vemepel have
Ginisun's experts, and one layer of each kind in turn; every second layer of Vemepel is dense). Run through ``bench.py --serving``.

Every kernel class is also timed (CUDA events around its launches, L2 flushed by the step's own traffic) against its roofline, the slower of algorithmic
bytes / measured copy bandwidth and FLOPs / measured bf16 GEMM rate. Times of single launches below ~5 us are dominated by launch overhead.
"""
from __future__ import annotations

import json
import statistics
from pathlib import Path

import torch

from ferrotorch_b200 import _lib
from ferrotorch_b200.models import GenerationConfig, LlamaConfig
from ferrotorch_b200.models.ginisun import GinisunConfig, GinisunModel, RandomGinisunWeights
from ferrotorch_b200.models.ginisun import ExpertConfig, MoeConfig
from ferrotorch_b200.models.mepupel import MepupelConfig, MepupelModel, RandomMepupelWeights
from ferrotorch_b200.models.pufevik import PufevikConfig, PufevikModel, RandomPufevikWeights
from ferrotorch_b200.models.vemepel import RandomVemepelWeights, VemepelConfig, VemepelModel
from ferrotorch_b200.models.llama_infer import LlamaTPEngine, TPContext
from ferrotorch_b200.models.serving import ServingEngine, StepEntry

SIZES = {
    "1k": dict(width=1024, heads=8, dim=64, rot_dim=32, vdim=64, kv_rank=256, experts=16, top=2, ff=1024, shared_ff=1024),
    "2k": dict(width=2048, heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, experts=64, top=6, ff=1408, shared_ff=2816),
    "4k": dict(width=4096, heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, experts=32, top=4, ff=2048, shared_ff=4096),
}
PUFEVIK = {                          # matrix memory beside the attention, window of its layers
    "1k": dict(memory_heads=4, memory_dim=128, memory_vdim=256, window=1024),
    "2k": dict(memory_heads=4, memory_dim=256, memory_vdim=512, window=1024),
    "4k": dict(memory_heads=8, memory_dim=256, memory_vdim=512, window=1024),
}
MEPUPEL = {                          # state space, groups of experts, latents
    "1k": dict(ssm=dict(heads=32, vdim=64, state=128, groups=1, norm_groups=1, conv=4), groups=4, keep=2, q_rank=512, kv_rank=256),
    "2k": dict(ssm=dict(heads=64, vdim=64, state=128, groups=8, norm_groups=8, conv=4), groups=8, keep=4, q_rank=1024, kv_rank=512),
    "4k": dict(ssm=dict(heads=128, vdim=64, state=128, groups=8, norm_groups=8, conv=4), groups=4, keep=2, q_rank=1536, kv_rank=512),
}
VOCAB = 32768


def peaks():
    p = Path(__file__).resolve().parents[1] / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def timed(fn, reps=7, warm=3):
    for _ in range(warm):
        fn()
    out = []
    for _ in range(reps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        out.append(e0.elapsed_time(e1))
    return statistics.median(out)


def kernel_table(fn, classify, roofs, bw, fl, reps=5):
    """us per call and roofline fraction by kernel class; ``roofs[label] = (bytes, flops)`` per call."""
    rows = {}
    for i in range(reps):
        _lib.trace_begin(classify)
        fn()
        for k, v in _lib.trace_end().items():
            rows.setdefault(k, []).append((v["ms"] * 1e3 / v["calls"], v["calls"]))
    out = {}
    for k, v in rows.items():
        us = statistics.median(x[0] for x in v)
        out[k] = {"us": round(us, 1), "calls": v[0][1]}
        if k in roofs:
            b, f = roofs[k]
            out[k]["roofline"] = round(max(b / bw, f / fl) * 1e6 / us, 3)
    return out


def _by_shape(names):
    """GEMM launches by (N, K) -> label, everything else by launcher name."""
    def c(fn, raw):
        if fn in ("ft_gemm_bf16", "ft_gemm_bf16_splitk"):
            o = 4 if fn == "ft_gemm_bf16" else 3
            return names.get((raw[o + 1], raw[o + 2]), f"gemm n={raw[o + 1]} k={raw[o + 2]}")
        if fn == "ft_gemm_grouped":
            return names.get(("grouped", raw[4], raw[5]), "grouped gemm")
        return names.get(fn, fn)
    return c


def run_ginisun(size, layers, batch, prompt, ctx, steps, kernels=True):
    bw, fl, _ = peaks()
    s = SIZES[size]
    cfg = GinisunConfig.uniform(layers, VOCAB, streams=4, **s)
    eng = ServingEngine(GinisunModel(cfg, RandomGinisunWeights(cfg)), max_tokens=max(batch * (ctx + steps * 4 + 64), prompt + 64), max_sequences=batch + 1)
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    def prefill():
        eng.step([StepEntry("p", ids, [prompt - 1])], ["p"])
    from ferrotorch_b200.models.serving import RowBatch
    eng._admit([StepEntry("p", ids, [prompt - 1])])
    rb = RowBatch([StepEntry("p", ids, [prompt - 1])], eng.cache, eng.device, eng.max_blocks)
    rb.tiles_for(eng.model.subs[0].attn.dims)
    device_prefill = lambda: eng.model.forward_rows(rb, eng.cache)          # the device part: tables of the batch are built once
    pre_ms, pre_e2e = timed(device_prefill), timed(lambda: (eng.release("p"), prefill()))
    W, H, T = s["width"], s["heads"], prompt
    D = eng.model.subs[0].attn.dims
    F, SF, E, top = s["ff"], s["shared_ff"], s["experts"], s["top"]
    nkv = H * (D.dim8 + D.v8)
    table = None
    if kernels:
        eng._admit([StepEntry("p", ids, [])])
        names = {(D.proj_cols, W): "projection gemm", (nkv, D.rank): "key/value expansion gemm", (W, H * D.v8): "output gemm", (E, W): "router gemm",
                 ("grouped", 2 * F, W): "experts gate/up gemm", ("grouped", W, F): "experts down gemm", (2 * SF, W): "shared gate/up gemm"}
        names[(W, SF)] = "output and shared down gemm" if SF == H * D.v8 else "shared down gemm"      # one shape: one label
        pairs = T * top
        def g_(n, k, out=2, m=T): return (2 * (m * k + n * k) + out * m * n, 2 * m * n * k)
        roofs = {"projection gemm": g_(D.proj_cols, W), "key/value expansion gemm": g_(nkv, D.rank), "output gemm": g_(W, H * D.v8, 4),
                 "experts gate/up gemm": (2 * (pairs * W + E * 2 * F * W + pairs * 2 * F), 4 * pairs * F * W), "experts down gemm": (2 * (pairs * W + E * F * W + pairs * F), 2 * pairs * F * W),
                 "shared gate/up gemm": g_(2 * SF, W), "shared down gemm": g_(W, SF, 4), "output and shared down gemm": g_(W, SF, 4),
                 "ft_latent_flash": (2 * T * (H * (D.dim8 + D.rot8) + nkv + H * D.v8), H * T * T * (D.dim + D.rot_dim + D.vdim)),
                 "ft_latent_prep": (2 * T * (2 * H * D.rot8 + D.rank + D.rot8 + 2 * D.row), 0),
                 "ft_moe_gather": (4 * pairs * W, 0), "ft_moe_act": ((pairs * F * 6 + T * SF * 6) / 2, 0)}
        # streams read and written in f32 (8 bytes each), bf16 operand out; attention adds one f32 plane, the mixture its bf16 rows (+ one f32 plane)
        roofs["ft_hyper_update"] = (T * W * (4 * 8 + 2 + (4 + (2 * top + (4 if SF else 0))) / 2), 0)
        table = kernel_table(device_prefill, _by_shape(names), roofs, bw, fl)
    eng.release("p")
    # decode
    seqs = [f"s{i}" for i in range(batch)]
    for q in seqs:
        eng.step([StepEntry(q, torch.randint(0, VOCAB, (ctx,), generator=g).tolist(), [])])
    eng.decode_greedy(seqs, [1] * batch, 4)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    best = []
    for _ in range(3):
        torch.cuda.synchronize()
        e0.record()
        eng.decode_greedy(seqs, [1] * batch, steps)
        e1.record()
        torch.cuda.synchronize()
        best.append(e0.elapsed_time(e1) / steps)
    dec_ms = statistics.median(best)
    dtable = None
    if kernels:
        eng.use_graph = False
        for q in seqs:
            eng.cache.reserve(q, eng.cache.lengths[q] + 1)
        eng.state.load([1 + i for i in range(batch)], [eng.cache.lengths[q] for q in seqs], eng.cache.block_table(seqs, eng.max_blocks))
        positions, lens = eng.state.positions.clone(), eng.state.seq_lens.clone()
        tokens = eng.state.tokens.clone()
        def one():
            eng.state.positions.copy_(positions); eng.state.seq_lens.copy_(lens); eng.state.tokens.copy_(tokens)
            eng.model.decode(eng.state, batch, eng.cache)
        one()
        active = int(eng.model._moe_buffers.n_active)               # experts in use (of the last layer; the layers are alike)
        L = eng.cache.lengths[seqs[0]] + 1
        names = {(D.proj_cols, W): "projection gemm", (W, H * D.v8): "output gemm", (VOCAB, W): "head gemm"}
        roofs = {"projection gemm": (2 * D.proj_cols * W, 0), "output gemm": (2 * H * D.v8 * W, 0), "head gemm": (2 * VOCAB * W, 0),
                 "ft_latent_decode": (2 * batch * L * D.row, 2 * batch * H * L * (D.row + D.r16)), "ft_latent_decode_prep": (2 * H * D.dim8 * D.rank, 0),
                 "ft_skinny_heads": (2 * H * D.v8 * D.rank, 0), "ft_moe_gate_up_small": (4 * W * (active * F + SF), 0), "ft_moe_down_small": (2 * W * (active * F + SF), 0),
                 "ft_hyper_update": (batch * W * 40, 0)}
        dtable = kernel_table(one, _by_shape(names), roofs, bw, fl)
        eng.use_graph = True
    eng.check()
    return {"prefill_ms": round(pre_ms, 3), "prefill_tokens_per_s": round(prompt / pre_ms * 1e3), "prefill_e2e_ms": round(pre_e2e, 3), "decode_ms_per_step": round(dec_ms, 4),
            "decode_tokens_per_s": round(batch / dec_ms * 1e3), "active_experts": active if kernels else None, "prefill_kernels": table,
            "decode_kernels": dtable}


def run_pufevik(size, layers, batch, prompt, ctx, steps, kernels=True):
    """Layers alternate: attention and matrix memory side by side, full attention."""
    bw, fl, _ = peaks()
    s, W = SIZES[size], SIZES[size]["width"]
    H, F = W // 128, s["top"] * s["ff"] + s["shared_ff"]
    G = max(1, H // 4)
    cfg = PufevikConfig.pattern(("pa" * layers)[:layers], VOCAB, W, F, H, G, 128, 128, **PUFEVIK[size])
    eng = ServingEngine(PufevikModel(cfg, RandomPufevikWeights(cfg)), max_tokens=max(batch * (ctx + steps * 4 + 64), prompt + 64), max_sequences=batch + 1)
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    from ferrotorch_b200.models.serving import RowBatch
    entry = [StepEntry("p", ids, [prompt - 1])]
    eng._admit(entry)
    rb = RowBatch(entry, eng.cache, eng.device, eng.max_blocks)
    device_prefill = lambda: eng.model.forward_rows(rb, eng.cache)          # the device part: tables of the batch are built once
    pre_ms = timed(device_prefill)
    par, att = eng.model.subs[0].mixer, eng.model.subs[2].mixer
    D, M = par.attn.dims, par.memory.dims
    T, win = prompt, D.window
    table = dtable = None
    def g_(n, k, out=2, m=T): return (2 * (m * k + n * k) + out * m * n, 2 * m * n * k)
    na, np_, n_gates = att.proj.shape[0], par.main, par.proj.shape[0] - par.main
    if kernels:
        names = {(np_, W): "projection gemm (two mixers)", (na, W): "projection gemm (attention)", (n_gates, W): "gate gemm", (W, par.out_cols): "output gemm (two mixers)",
                 (W, att.out_cols): "output gemm (attention)", (2 * F, W): "gate/up gemm", (W, F): "down gemm"}
        classify = _by_shape(names)
        seen = win * T - win * (win - 1) // 2 if win < T else T * (T + 1) // 2            # keys that the window's queries see
        qkv = D.qkv_cols
        roofs = {"projection gemm (two mixers)": g_(np_, W), "projection gemm (attention)": g_(na, W), "gate gemm": g_(n_gates, W, 4), "output gemm (two mixers)": g_(W, par.out_cols, 4),
                 "output gemm (attention)": g_(W, att.out_cols, 4), "gate/up gemm": g_(2 * F, W), "down gemm": g_(W, F, 4),
                 "flash (window)": (2 * T * (qkv + D.out_cols), 4 * H * seen * 128), "flash (full)": (2 * T * (qkv + 2 * D.out_cols), H * T * T * 256),
                 "ft_gqa_prep": (2 * T * (2 * qkv), 0), "ft_gated_act": (6 * T * F, 0), "ft_residual_update": (14 * T * W, 0),
                 # inner: keys and values in; outputs: queries, keys, values in, f32 outputs out; finish: those, gates in, bf16 out. Products of a chunk of 64
                 "memory walk (states)": (2 * T * M.heads * (M.d16 + M.v16), 2 * T * M.heads * M.d16 * M.v16),
                 "memory walk (outputs)": (T * M.heads * (4 * M.d16 + 6 * M.v16), 2 * T * M.heads * (2 * M.d16 * M.v16 + 32 * (M.d16 + M.v16))),
                 "ft_mm_finish": (T * M.heads * M.v16 * 8, 0)}
        def label(fn, raw):
            if fn == "ft_gqa_flash":
                return "flash (window)" if raw[15] else "flash (full)"
            if fn == "ft_mm_walk":
                return "memory walk (outputs)" if raw[17] else "memory walk (states)"
            return classify(fn, raw)
        table = kernel_table(device_prefill, label, roofs, bw, fl)
    eng.release("p")
    seqs = [f"s{i}" for i in range(batch)]
    for q in seqs:
        eng.step([StepEntry(q, torch.randint(0, VOCAB, (ctx,), generator=g).tolist(), [])])
    eng.decode_greedy(seqs, [1] * batch, 4)
    best = []
    for _ in range(3):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        eng.decode_greedy(seqs, [1] * batch, steps)
        e1.record()
        torch.cuda.synchronize()
        best.append(e0.elapsed_time(e1) / steps)
    dec_ms = statistics.median(best)
    if kernels:
        for q in seqs:
            eng.cache.reserve(q, eng.cache.lengths[q] + 1)
        eng._load_state(seqs, [1 + i for i in range(batch)])
        positions, lens, tokens = eng.state.positions.clone(), eng.state.seq_lens.clone(), eng.state.tokens.clone()
        def one():
            eng.state.positions.copy_(positions); eng.state.seq_lens.copy_(lens); eng.state.tokens.copy_(tokens)
            eng.model.decode(eng.state, batch, eng.cache)
        one()
        L = eng.cache.lengths[seqs[0]] + 1
        names = {(par.proj.shape[0], W): "projection gemm (two mixers)", (na, W): "projection gemm (attention)", (W, par.out_cols): "output gemm (two mixers)",
                 (W, att.out_cols): "output gemm (attention)", (2 * F, W): "gate/up gemm", (W, F): "down gemm", (VOCAB, W): "head gemm"}
        classify = _by_shape(names)
        roofs = {"projection gemm (two mixers)": (2 * par.proj.shape[0] * W, 0), "projection gemm (attention)": (2 * na * W, 0), "output gemm (two mixers)": (2 * W * par.out_cols, 0),
                 "output gemm (attention)": (2 * W * att.out_cols, 0), "gate/up gemm": (4 * F * W, 0), "down gemm": (2 * F * W, 0), "head gemm": (2 * VOCAB * W, 0),
                 "attention (window)": (2 * batch * min(L, win) * D.row, 0), "attention (full)": (2 * batch * L * D.row, 0), "ft_mm_decode": (2 * batch * M.state_size * 4, 0)}
        def label_d(fn, raw):
            if fn == "ft_gqa_decode":
                return "attention (window)" if raw[12] else "attention (full)"
            return classify(fn, raw)
        dtable = kernel_table(one, label_d, roofs, bw, fl)
    eng.check()
    return {"prefill_ms": round(pre_ms, 3), "prefill_tokens_per_s": round(prompt / pre_ms * 1e3), "decode_ms_per_step": round(dec_ms, 4),
            "decode_tokens_per_s": round(batch / dec_ms * 1e3), "prefill_kernels": table, "decode_kernels": dtable}


def run_mepupel(size, layers, batch, prompt, ctx, steps, kernels=True):
    """Layers in turn: state space, windowed attention, latent attention, latent attention on the latent before it; experts in every layer."""
    from ferrotorch_b200.models.serving import RowBatch
    bw, fl, _ = peaks()
    s, e = SIZES[size], MEPUPEL[size]
    W, T, F, SF, E, top = s["width"], prompt, s["ff"], s["shared_ff"], s["experts"], s["top"]
    H = W // 128
    G = max(1, H // 4)
    att = dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, rot=dict(base=1e4, dims=64, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0)),
               mask=dict(size=1024, keep_first=64))
    lat = dict(heads=H, dim=128, vdim=128, q_rank=e["q_rank"], kv_rank=e["kv_rank"], scale=128 ** -0.5)
    cfg = MepupelConfig.pattern(("mals" * layers)[:layers], VOCAB, W, e["ssm"], att, lat,
                                MoeConfig(E, top, ExpertConfig(F), ExpertConfig(SF), e["groups"], e["keep"], 2.0), residual_mult=0.5)
    eng = ServingEngine(MepupelModel(cfg, RandomMepupelWeights(cfg)), max_tokens=max(batch * (ctx + steps * 4 + 64), prompt + 64), max_sequences=batch + 1)
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    entry = [StepEntry("p", ids, [prompt - 1])]
    eng._admit(entry)
    rb = RowBatch(entry, eng.cache, eng.device, eng.max_blocks)
    device_prefill = lambda: eng.model.forward_rows(rb, eng.cache)          # the device part: tables of the batch are built once
    pre_ms = timed(device_prefill)
    by = {k: next((l for l in eng.model.layers if getattr(l, k)), None) for k in ("ssm", "attn", "latent")}
    S, A, L = (by[k].mixer.dims if by[k] else None for k in ("ssm", "attn", "latent"))
    table = dtable = None
    def g_(n, k, out=2, m=T): return (2 * (m * k + n * k) + out * m * n, 2 * m * n * k)
    pairs, nkv = T * top, H * (L.dim8 + L.v8)
    common = {(S.main, W): "projection gemm (state space)", (by["attn"].proj.shape[0], W): "projection gemm (attention)", (L.proj_cols, W): "projection gemm (latent)",
              (L.q_cols, W): "projection gemm (latent, shared)", (H * L.dim8, L.q_rank): "query expansion gemm", (W, S.out_cols): "output gemm (state space)",
              (2 * SF, W): "shared gate/up gemm", ("grouped", 2 * F, W): "experts gate/up gemm", ("grouped", W, F): "experts down gemm"}
    if kernels:
        names = dict(common)
        names.update({(S.h8, W): "step size gemm", (nkv, L.rank): "key/value expansion gemm", (E, W): "router gemm"})
        for shape, label in (((W, A.out_cols), "output gemm (attention)"), ((W, SF), "shared down gemm")):
            names[shape] = "output gemms and shared down gemm" if SF in (A.out_cols, S.out_cols) and shape[1] == SF else label      # one shape: one label
        classify = _by_shape(names)
        win, keep = A.window, A.keep
        seen = win * T - win * (win - 1) // 2 + keep * max(0, T - win) if win < T else T * (T + 1) // 2
        N = S.n16
        roofs = {names[k]: g_(k[0], k[1], 4 if "output" in names[k] or "down" in names[k] or "step" in names[k] or "router" in names[k] else 2) for k in names if k[0] != "grouped"}
        roofs.update({
            "experts gate/up gemm": (2 * (pairs * W + E * 2 * F * W + pairs * 2 * F), 4 * pairs * F * W), "experts down gemm": (2 * (pairs * W + E * F * W + pairs * F), 2 * pairs * F * W),
            "ft_gqa_flash": (2 * T * (A.qkv_cols + A.out_cols), 4 * H * seen * 128), "ft_gqa_prep": (4 * T * (H * A.rot_dims + A.qkv_cols - A.k_col), 0),
            "ft_latent_flash": (2 * T * (H * L.dim8 + nkv + H * L.v8), H * T * T * (L.dim + L.vdim)), "ft_latent_prep": (2 * T * (2 * L.q_rank + L.rank + 2 * L.row), 0),
            "ft_moe_gather": (4 * pairs * W, 0), "ft_moe_act": ((pairs * F * 6 + T * SF * 6) / 2, 0), "ft_moe_topk": (T * E * 4, 0),
            "ft_parallel_update": (T * W * (8 + 4 + 4 + 2 * top + 4), 0), "ft_ssm_conv": (4 * T * S.channels, 0), "ft_ssm_finish": (6 * T * S.out_cols, 0),
            "state walk (outputs)": (2 * T * (S.channels + S.out_cols), 2 * T * S.heads * (2 * N * S.v16 + 32 * (N + S.v16))),
            "state walk (states)": (2 * T * (S.channels - S.groups * N), 2 * T * S.heads * N * S.v16)})
        def label(fn, raw):
            if fn == "ft_ssm_walk":
                return "state walk (outputs)" if raw[17] else "state walk (states)"
            return classify(fn, raw)
        table = kernel_table(device_prefill, label, roofs, bw, fl)
    eng.release("p")
    seqs = [f"s{i}" for i in range(batch)]
    for q in seqs:
        eng.step([StepEntry(q, torch.randint(0, VOCAB, (ctx,), generator=g).tolist(), [])])
    eng.decode_greedy(seqs, [1] * batch, 4)
    best = []
    for _ in range(3):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        eng.decode_greedy(seqs, [1] * batch, steps)
        e1.record()
        torch.cuda.synchronize()
        best.append(e0.elapsed_time(e1) / steps)
    dec_ms = statistics.median(best)
    active = None
    if kernels:
        for q in seqs:
            eng.cache.reserve(q, eng.cache.lengths[q] + 1)
        eng._load_state(seqs, [1 + i for i in range(batch)])
        positions, lens, tokens = eng.state.positions.clone(), eng.state.seq_lens.clone(), eng.state.tokens.clone()
        def one():
            eng.state.positions.copy_(positions); eng.state.seq_lens.copy_(lens); eng.state.tokens.copy_(tokens)
            eng.model.decode(eng.state, batch, eng.cache)
        one()
        active = int(eng.model._moe_buffers.n_active)               # experts in use (of the last layer; the layers are alike)
        eng.model.side_by_side = False                              # kernels one by one
        n = eng.cache.lengths[seqs[0]] + 1
        names = dict(common)
        names.update({(S.main + S.h8, W): "projection gemm (state space)", (W, A.out_cols): "output gemm (attention)", (VOCAB, W): "head gemm"})
        roofs = {names[k]: (2 * k[0] * k[1], 0) for k in names if k[0] != "grouped"}
        roofs.update({"ft_gqa_decode": (2 * batch * min(n, A.window + A.keep) * A.row, 0), "ft_latent_decode": (2 * batch * n * L.row, 2 * batch * H * n * (L.row + L.r16)),
                      "ft_latent_decode_prep": (2 * H * L.dim8 * L.rank, 0), "ft_skinny_heads": (2 * H * L.v8 * L.rank, 0), "ft_ssm_decode": (8 * batch * S.state_size, 0),
                      "ft_moe_gate_up_small": (4 * W * (active * F + SF), 0), "ft_moe_down_small": (2 * W * (active * F + SF), 0), "ft_parallel_update": (batch * W * (12 + 4 * (top + 1) + 16), 0)})
        dtable = kernel_table(one, _by_shape(names), roofs, bw, fl)
    eng.check()
    return {"prefill_ms": round(pre_ms, 3), "prefill_tokens_per_s": round(prompt / pre_ms * 1e3), "decode_ms_per_step": round(dec_ms, 4), "decode_tokens_per_s": round(batch / dec_ms * 1e3),
            "active_experts": active, "prefill_kernels": table, "decode_kernels": dtable}


def run_vemepel(size, layers, batch, prompt, ctx, steps, kernels=True):
    """Layers in turn: differential attention in chunks, latent attention with a rotated part, without positions, differential attention on the first one's keys and values; dense
    and mixture-of-experts feed-forwards alternate."""
    from ferrotorch_b200.models.serving import RowBatch
    bw, fl, _ = peaks()
    s = SIZES[size]
    W, T, F, E, top, R = s["width"], prompt, s["ff"], s["experts"], s["top"], s["kv_rank"]
    H, DF = W // 128, top * F + s["shared_ff"]
    G = max(1, H // 4)
    chunk = 1280                                        # not a divisor of the context: the decoded tokens' chunk is three quarters full
    att = dict(heads=H, kv_heads=G, dim=64, vdim=128, scale=64 ** -0.5, diff=0.5, mask=dict(size=chunk))
    lat = dict(heads=H, dim=128, vdim=128, kv_rank=R, scale=128 ** -0.5)
    cfg = VemepelConfig.pattern(("arls" * layers)[:layers], VOCAB, W, att, lat, dict(lat, rot_dim=64, rot=dict(base=1e4, dims=64)), MoeConfig(E, top, ExpertConfig(F)), dense_ff=DF)
    eng = ServingEngine(VemepelModel(cfg, RandomVemepelWeights(cfg)), max_tokens=max(batch * (ctx + steps * 4 + 64), prompt + 64), max_sequences=batch + 1)
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    entry = [StepEntry("p", ids, [prompt - 1])]
    eng._admit(entry)
    rb = RowBatch(entry, eng.cache, eng.device, eng.max_blocks)
    device_prefill = lambda: eng.model.forward_rows(rb, eng.cache)          # the device part: tables of the batch are built once
    pre_ms = timed(device_prefill)
    A = next(l.attn.dims for l in eng.model.layers if l.attn)
    P, L = (next((l.latent.dims for l in eng.model.layers if l.latent and bool(l.latent.dims.rot_dim) == rotated), None) for rotated in (True, False))
    n_layers, pairs, nkv = len(eng.model.layers), T * top, H * (L.dim8 + L.v8)
    deep = sum(range(1, n_layers + 1)) / n_layers                           # results that an average reads, over the layers
    common = {(A.qkv_cols, W): "projection gemm (attention)", (A.k_col, W): "projection gemm (attention, shared keys)", (P.proj_cols, W): "projection gemm (latent, rotated)",
              (L.proj_cols, W): "projection gemm (latent)", (W, A.out_cols): "output gemm", (DF, W): "up gemm", (W, DF): "down gemm",
              ("grouped", 2 * F, W): "experts gate/up gemm", ("grouped", W, F): "experts down gemm"}
    table = dtable = active = None
    def g_(n, k, out=2, m=T): return (2 * (m * k + n * k) + out * m * n, 2 * m * n * k)
    if kernels:
        names = dict(common)
        names.update({(nkv, R): "key/value expansion gemm", (E, W): "router gemm"})
        seen = sum(min(i % chunk, chunk) + 1 for i in range(T))             # keys that the chunks' queries see
        roofs = {names[k]: g_(k[0], k[1], 4 if "output" in names[k] or "down" in names[k] or "router" in names[k] else 2) for k in names if k[0] != "grouped"}
        roofs.update({
            "experts gate/up gemm": (2 * (pairs * W + E * 2 * F * W + pairs * 2 * F), 4 * pairs * F * W), "experts down gemm": (2 * (pairs * W + E * F * W + pairs * F), 2 * pairs * F * W),
            "ft_gqa_flash": (2 * T * (A.qkv_cols + A.out_cols), 2 * 2 * H * seen * (A.dim + A.vdim)), "ft_gqa_prep": (4 * T * (A.qkv_cols - A.k_col), 0),
            "flash (latent, rotated)": (2 * T * (H * (P.dim8 + P.rot8) + nkv + 2 * H * P.v8), H * T * T * (P.dim + P.rot_dim + P.vdim)),
            "flash (latent)": (2 * T * (H * L.dim8 + nkv + H * L.v8), H * T * T * (L.dim + L.vdim)),
            "prep (latent, rotated)": (2 * T * (2 * H * P.rot8 + R + P.rot8 + 2 * P.row), 0), "prep (latent)": (2 * T * (R + 2 * L.row), 0),
            "ft_moe_gather": (4 * pairs * W, 0), "ft_moe_act": (pairs * F * 6, 0), "ft_moe_topk": (T * E * 4, 0), "ft_poly_norm": (4 * T * DF, 0), "ft_token_shift": (6 * T * W, 0),
            "ft_residual_update": (T * W * 14, 0), "ft_depth_update": (T * W * (4 * deep + 12 + (4 + 2 * top) / 2), 0), "ft_depth_embed": (T * W * 10, 0)})
        classify = _by_shape(names)
        def label(fn, raw):
            if fn == "ft_latent_flash":
                return "flash (latent, rotated)" if raw[12] else "flash (latent)"
            if fn == "ft_latent_prep":
                return "prep (latent, rotated)" if raw[5] else "prep (latent)"
            return classify(fn, raw)
        table = kernel_table(device_prefill, label, roofs, bw, fl)
    eng.release("p")
    seqs = [f"s{i}" for i in range(batch)]
    for q in seqs:
        eng.step([StepEntry(q, torch.randint(0, VOCAB, (ctx,), generator=g).tolist(), [])])
    eng.decode_greedy(seqs, [1] * batch, 4)
    best = []
    for _ in range(3):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        eng.decode_greedy(seqs, [1] * batch, steps)
        e1.record()
        torch.cuda.synchronize()
        best.append(e0.elapsed_time(e1) / steps)
    dec_ms = statistics.median(best)
    if kernels:
        for q in seqs:
            eng.cache.reserve(q, eng.cache.lengths[q] + 1)
        eng._load_state(seqs, [1 + i for i in range(batch)])
        positions, lens, tokens = eng.state.positions.clone(), eng.state.seq_lens.clone(), eng.state.tokens.clone()
        def one():
            eng.state.positions.copy_(positions); eng.state.seq_lens.copy_(lens); eng.state.tokens.copy_(tokens)
            eng.model.decode(eng.state, batch, eng.cache)
        one()
        active = int(eng.model._moe_buffers.n_active)               # experts in use (of the last layer; the layers are alike)
        n = eng.cache.lengths[seqs[0]] + 1
        names = dict(common)
        names[(VOCAB, W)] = "head gemm"
        roofs = {names[k]: (2 * k[0] * k[1], 0) for k in names if k[0] != "grouped"}
        roofs.update({"ft_gqa_decode": (2 * batch * ((n - 1) % chunk + 1) * A.row, 0),
                      "attention (latent, rotated)": (2 * batch * n * P.row, 2 * batch * H * n * (P.row + P.r16)), "attention (latent)": (2 * batch * n * L.row, 2 * batch * H * n * (L.row + L.r16)),
                      "ft_latent_decode_prep": (2 * H * L.dim8 * R, 0), "ft_skinny_heads": (2 * H * L.v8 * R, 0), "ft_moe_gate_up_small": (4 * W * active * F, 0),
                      "ft_moe_down_small": (2 * W * active * F, 0)})
        classify_d = _by_shape(names)
        def label_d(fn, raw):
            if fn == "ft_latent_decode":
                return "attention (latent, rotated)" if raw[7] else "attention (latent)"
            return classify_d(fn, raw)
        dtable = kernel_table(one, label_d, roofs, bw, fl)
    eng.check()
    return {"prefill_ms": round(pre_ms, 3), "prefill_tokens_per_s": round(prompt / pre_ms * 1e3), "decode_ms_per_step": round(dec_ms, 4), "decode_tokens_per_s": round(batch / dec_ms * 1e3),
            "active_experts": active, "prefill_kernels": table, "decode_kernels": dtable}


def run_llama(size, layers, batch, prompt, ctx, steps, kernels=True):
    bw, fl, _ = peaks()
    s = SIZES[size]
    W, H = s["width"], s["width"] // 128
    kvh = max(1, H // 4)
    F = s["top"] * s["ff"] + s["shared_ff"]
    cfg = LlamaConfig(vocab_size=VOCAB, hidden_size=W, intermediate_size=F, num_hidden_layers=layers, num_attention_heads=H, num_key_value_heads=kvh)
    g = torch.Generator().manual_seed(1)
    eng = LlamaTPEngine(cfg, TPContext("cuda"), max_batch=1, max_seq=prompt + 16)
    ids = torch.randint(0, VOCAB, (1, prompt), generator=g).cuda()
    pre_ms = timed(lambda: eng.prefill(ids))
    T, nq = prompt, (H + 2 * kvh) * 128
    table = dtable = None
    def g_(n, k, m=T): return (2 * (m * k + n * k + m * n), 2 * m * n * k)
    if kernels:
        names = {(nq, W): "qkv gemm", (W, H * 128): "output gemm", (2 * F, W): "gate/up gemm", (W, F): "down gemm"}
        roofs = {"qkv gemm": g_(nq, W), "output gemm": g_(W, H * 128), "gate/up gemm": g_(2 * F, W), "down gemm": g_(W, F),
                 "ft_flash_fwd": (2 * T * (nq + H * 128), H * T * T * 256), "ft_rmsnorm_fwd": (6 * T * W, 0), "ft_swiglu_fwd": (6 * T * F, 0), "ft_add_bf16": (6 * T * W, 0),
                 "ft_rope_inplace": (4 * T * (H + kvh) * 128, 0)}
        table = kernel_table(lambda: eng.prefill(ids), _by_shape(names), roofs, bw, fl)
    del eng
    torch.cuda.empty_cache()
    eng = LlamaTPEngine(cfg, TPContext("cuda"), max_batch=batch, max_seq=ctx + 4 * steps + 64)
    eng.prefill(torch.randint(0, VOCAB, (batch, ctx), generator=g).cuda())
    for _ in range(4):
        eng.decode_step()
    best = []
    for _ in range(3):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for _ in range(steps):
            eng.decode_step()
        e1.record()
        torch.cuda.synchronize()
        best.append(e0.elapsed_time(e1) / steps)
    dec_ms = statistics.median(best)
    if kernels:
        L = ctx + 4
        names = {(nq, W): "qkv gemm", (W, H * 128): "output gemm", (2 * F, W): "gate/up gemm", (W, F): "down gemm", (VOCAB, W): "head gemm"}
        roofs = {"qkv gemm": (2 * nq * W, 0), "output gemm": (2 * W * H * 128, 0), "gate/up gemm": (4 * F * W, 0), "down gemm": (2 * F * W, 0), "head gemm": (2 * VOCAB * W, 0),
                 "ft_paged_attn_decode": (4 * batch * L * kvh * 128, 0)}
        eng.use_graph = False
        import os
        os.environ["FT_DECODE_PDL"] = "0"
        dtable = kernel_table(lambda: eng.decode_step(), _by_shape(names), roofs, bw, fl)
        os.environ.pop("FT_DECODE_PDL")
    eng.check()
    return {"prefill_ms": round(pre_ms, 3), "prefill_tokens_per_s": round(prompt / pre_ms * 1e3), "decode_ms_per_step": round(dec_ms, 4),
            "decode_tokens_per_s": round(batch / dec_ms * 1e3), "prefill_kernels": table, "decode_kernels": dtable}


def main(sizes="1k,2k,4k", layers=4, batch=8, prompt=4096, ctx=2048, steps=64, kernels=True, models="") -> int:
    torch.cuda.set_device(0)
    _, _, of = peaks()
    res = {}
    for size in sizes.split(","):
        res[size] = {}
        for name, run in (("ginisun", run_ginisun), ("pufevik", run_pufevik), ("mepupel", run_mepupel), ("vemepel", run_vemepel), ("llama", run_llama)):
            if models and name not in models.split(","):
                continue
            res[size][name] = run(size, layers, batch, prompt, ctx, steps, kernels)
            torch.cuda.empty_cache()
    print(json.dumps({"bench": "serving", "layers": layers, "decode_batch": batch, "prompt": prompt, "context": ctx, "dtype": "bf16", "peaks": of,
                      "data": "synthetic (uniform random token ids, random weights)", "sizes": res, "kernel_status": _lib.read_status()}))
    return 0
