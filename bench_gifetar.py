"""Gifetar layers beside DecoderStack layers of equal size (`python bench.py --micro gifetar`).

Equal size: the same width, heads, kv heads, cache bytes per token (two maps of 64 + a value of 128 against a key and
a value of 128), and as many feed-forward parameters per token (top x ff against the dense inner size).  Random
weights, synthetic tokens and caches.  For each size: throughput of a prompt and of a decode step through Engine's
model calls, and each kernel alone -- with its time, its roofline time (the larger of flops / matrix peak and bytes /
copy peak) and how many times longer it takes -- beside the like kernel of the other model.

Kernels are timed with CUDA events on their stream, a write of 256 MB (twice the L2) in front of every call, median of
the calls; the steps without a flush (their weights and caches exceed the L2)."""
from __future__ import annotations

import json
import os

import torch

ROOT = os.path.dirname(os.path.abspath(__file__))

SIZES = {
    # width, heads, kv heads, experts, top, ff | prompt tokens, decode batch, context
    "w2048": dict(width=2048, heads=16, kv_heads=4, experts=64, top=8, ff=768, prompt=8192, batch=64, ctx=8192),
    "w4096": dict(width=4096, heads=32, kv_heads=8, experts=32, top=4, ff=2048, prompt=8192, batch=128, ctx=4096),
}
LAYERS, VOCAB, DIM, VDIM = 2, 32768, 64, 128


def _peaks():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]) * 1e9, float(p["bf16_tflops"]) * 1e12, "measured"
    except Exception:
        return 6650e9, 1590e12, "fallback"


class Timer:
    def __init__(self, device, iters):
        self.flush = torch.empty(64 << 20, dtype=torch.float32, device=device)
        self.iters = iters

    def __call__(self, fn, before=None):
        for _ in range(3):
            if before:
                before()
            fn()
        pairs = []
        for _ in range(self.iters):
            self.flush.fill_(0.0)
            if before:
                before()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            pairs.append((a, b))
        torch.cuda.synchronize()
        ms = sorted(a.elapsed_time(b) for a, b in pairs)
        return ms[len(ms) // 2] * 1e3                        # microseconds


def _step_ms(fn, iters):
    for _ in range(3):
        fn()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def run(args, clock_sampler):
    import kinetics_b200 as kb
    from kinetics_b200 import layer_ops as lo, ops
    from kinetics_b200.gifetar import Gifetar, GifetarConfig, GifetarLayer, random_weights

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    hbm, mm, peak_of = _peaks()
    timer = Timer(dev, max(3, min(args.steps, 20)))
    only = args.only_kernel
    sampler = clock_sampler(0)
    result = {"micro": "gifetar", "peaks": {"bytes_per_s": hbm, "flops_per_s": mm, "of": peak_of},
              "l2": "256 MB written in front of every kernel call; steps exceed the L2", "layers": LAYERS, "vocab": VOCAB,
              "sizes": {}}
    launches0 = ops.launch_count()

    def record(table, name, us, flop=0.0, nbytes=0.0):
        roof = max(flop / mm, nbytes / hbm) * 1e6
        table[name] = {"us": round(us, 2), "roofline_us": round(roof, 2), "times_roofline": round(us / roof, 2),
                       "bound": "matrix" if flop / mm > nbytes / hbm else "hbm"}

    with sampler:
        for size, z in SIZES.items():
            C, H, G, E, T, F = (z[k] for k in ("width", "heads", "kv_heads", "experts", "top", "ff"))
            layer = GifetarLayer(heads=H, kv_heads=G, dim=DIM, vdim=VDIM, scale=DIM ** -0.5, softcap=30.0, diff=0.3,
                                 temp_coef=0.1, temp_every=2048, experts=E, top=T, ff=F)
            gc = GifetarConfig(vocab=VOCAB, width=C, norm_eps=1e-6, residual_mult=0.3, layers=(layer,) * LAYERS)
            sc = kb.LayerConfig(hidden_size=C, num_attention_heads=H, num_key_value_heads=G, intermediate_size=T * F,
                                num_hidden_layers=LAYERS, vocab_size=VOCAB)
            n, B, ctx = z["prompt"], z["batch"], z["ctx"]
            out = {"config": dict(z, dim=DIM, vdim=VDIM, dense_inner=T * F), "prefill": {}, "decode": {}}
            gif = Gifetar(gc, random_weights(gc, args.seed, dev), dev)
            stack = kb.DecoderStack(sc, dev, max_positions=max(n, ctx) + 256, seed=args.seed, decode_batch=B)
            tokens = torch.randint(0, VOCAB, (1, n), device=dev)
            pos = torch.arange(n, device=dev)[None]
            slot0 = torch.tensor([0], device=dev)

            # ---------------- whole steps
            def engine(model, kv, lens):
                kv.assume_filled({s: lens for s in range(B)}, headroom=200)
                e = kb.Engine(model, kv, lens + 256, dev, repeat_check=False)
                for s in range(B):
                    e.slots_occupy_status[s] = True
                    e._offsets_host[s] = e._prompt_host[s] = lens
                e.slots_offsets.fill_(lens)
                e.slots_tokens.random_(0, VOCAB)
                return e

            def managers(model, batch, length):
                if model is gif:
                    return gif.new_cache(batch, length + 256, batch * ((length + 255) // 64 + 1))
                return kb.PooledKVManager(sc, batch, length + 256, dev, torch.bfloat16,
                                          num_pages=batch * ((length + 255) // 16 + 3))

            steps = {}
            if not only:
                for name, model in (("gifetar", gif), ("decoder_stack", stack)):
                    kv = managers(model, 1, n)

                    def prompt():
                        kv.clear_cache(0)
                        kv.admit(0, n, n)
                        kv.begin_step([0])
                        model.next_tokens(tokens, pos, slot0, kv, last_only=True)
                    ms = _step_ms(prompt, 5)
                    kv.check_status()
                    del kv
                    kv = managers(model, B, ctx)
                    for t in (kv.k_pages + kv.v_pages if model is gif else kv.kv_pages):
                        t.normal_()
                    eng = engine(model, kv, ctx)
                    slots = list(range(B))
                    ms_d = _step_ms(lambda: eng.decode_graphed(slots), 30)
                    kv.check_status()
                    model.check_status()
                    steps[name] = {"prefill_ms": ms, "prefill_tokens_per_s": n / ms * 1e3, "decode_ms": ms_d,
                                   "decode_tokens_per_s": B / ms_d * 1e3}
                    eng._graph = None
                    del eng, kv
                out["steps"] = steps

            # ---------------- kernel by kernel
            gen = torch.Generator(device=dev).manual_seed(args.seed)
            rnd = lambda *s: torch.randn(*s, device=dev, generator=gen).to(torch.bfloat16)
            L, SL = gif.layers[0], stack.layers[0]
            spec, moe = L["spec"], L["moe"]

            def want(name):
                return only in name

            for phase, rows in (("prefill", n), ("decode", B)):
                ours, like = {}, {}
                batch, length = (1, n) if phase == "prefill" else (B, ctx)
                h, y = rnd(rows, C), rnd(rows, C)
                x = torch.randn(rows, C, device=dev)
                proj = rnd(rows, spec.q_cols + spec.k_cols + spec.v_cols)
                attn = rnd(rows, spec.o_cols)
                ps = 64
                pages = (length + ps - 1) // ps
                i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
                perm = torch.randperm(batch * pages, device=dev, generator=gen).to(torch.int32)
                table = lo.PageTable(perm, i32([i * pages for i in range(batch + 1)]),
                                     i32([length - (pages - 1) * ps] * batch), ps, batch * pages)
                kp, vp = rnd(batch * pages, G * 2, ps, DIM), rnd(batch * pages, G, ps, VDIM)
                indptr = i32([0, n]) if phase == "prefill" else None
                splits = lo.attention_splits(spec, batch, length, torch.bfloat16)
                keys = n * (n + 1) / 2 if phase == "prefill" else batch * length
                kv_bytes = batch * length * G * (2 * DIM + VDIM) * 2
                io = rows * (spec.q_cols + spec.o_cols) * 2
                if want("attention"):
                    us = timer(lambda: lo.paged_attention(proj, kp, vp, table, spec, indptr, n, splits))
                    record(ours, "attention", us, keys * H * 4 * (DIM + VDIM), kv_bytes + io)
                    p16 = (length + 15) // 16
                    cache = rnd(batch * p16, 2, 16, G, 128)
                    perm16 = torch.randperm(batch * p16, device=dev, generator=gen).to(torch.int32)
                    ptr16, last16 = i32([i * p16 for i in range(batch + 1)]), i32([length - (p16 - 1) * 16] * batch)
                    q = rnd(rows, H, 128)
                    if phase == "prefill":
                        us = timer(lambda: ops.prefill_attention(q, indptr, n, cache, perm16, ptr16, last16))
                    else:
                        us = timer(lambda: ops.dense_decode(q, cache, perm16, ptr16, last16, p16))
                    record(like, "attention", us, keys * H * 4 * 128, batch * length * G * 256 * 2 + 2 * rows * H * 128 * 2)
                    del cache
                if want("append"):
                    us = timer(lambda: lo.kv_append(proj, spec.q_cols, spec.q_cols + spec.k_cols, kp, vp, table, spec, indptr))
                    record(ours, "append", us, 0, 2 * rows * (spec.k_cols + spec.v_cols) * 2)
                    p16 = (length + 15) // 16
                    cache = rnd(batch * p16, 2, 16, G, 128)
                    perm16 = torch.randperm(batch * p16, device=dev, generator=gen).to(torch.int32)
                    ptr16, last16 = i32([i * p16 for i in range(batch + 1)]), i32([length - (p16 - 1) * 16] * batch)
                    k16, v16 = rnd(rows, G, 128), rnd(rows, G, 128)
                    ap = indptr if phase == "prefill" else i32(list(range(batch + 1)))
                    us = timer(lambda: ops.append_tokens(k16, v16, ap, cache, None, perm16, ptr16, last16))
                    record(like, "append", us, 0, 2 * rows * G * 256 * 2)
                    del cache
                del kp, vp
                if want("row_norms"):
                    us = timer(lambda: lo.residual_norm(x, h, C, 1e-6, pre=L["norm2"], y=y, post=L["norm1b"], mult=0.3))
                    record(ours, "row_norms", us, 0, rows * C * (2 + 2 + 4 + 4))
                    us = timer(lambda: ops.add_rmsnorm(y, h, SL["post_norm"], 1e-6))
                    record(like, "row_norms", us, 0, rows * C * 8)
                    parts = rnd(rows, T, C)
                    us = timer(lambda: lo.residual_norm(x, h, C, 1e-6, pre=L["norm1"], y=parts, parts=T, post=L["norm2b"],
                                                        mult=0.3))
                    record(ours, "row_norms_of_expert_parts", us, 0, rows * C * (2 * T + 2 + 4 + 4))
                    del parts
                h = rnd(rows, C)
                if want("router"):
                    us = timer(lambda: lo.moe_route(h, L["router"], L["router_b"], moe, L["counts"]),
                               before=lambda: L["counts"].zero_())
                    record(ours, "router", us, 2.0 * rows * E * C, rows * C * 2 + E * C * 2 + rows * T * 12)
                if want("expert"):
                    L["counts"].zero_()
                    r = lo.moe_route(h, L["router"], L["router_b"], moe, L["counts"])
                    used = int((r.counts > 0).sum())
                    lib, m = kb._lib.load_layers(), moe.c(1)
                    import ctypes
                    act, part = rnd(rows * T, F), rnd(rows, T, C)

                    def gemm(stage, src, w, dst):
                        kb._lib.check_layers(lib.ktk_moe_gemm(stage, ops._ptr(src), ops._ptr(w), ops._ptr(dst),
                                                              ops._ptr(r.weights), ops._ptr(r.counts), ops._ptr(r.bucket),
                                                              rows, ctypes.byref(m), 0, ops._ptr(gif.status), ops._stream()))
                    us = timer(lambda: gemm(0, h, L["gate_up"], act))
                    record(ours, "expert_gate_up", us, 4.0 * rows * T * C * F, used * 2 * C * F * 2 + rows * (C + T * F) * 2)
                    us = timer(lambda: gemm(1, act, L["down"], part))
                    record(ours, "expert_down", us, 2.0 * rows * T * C * F, used * C * F * 2 + rows * T * (F + C) * 2)
                    gu = torch.empty(rows, 2 * T * F, dtype=torch.bfloat16, device=dev)

                    def dense_gate_up():
                        torch.mm(h, SL["gate_up"].t(), out=gu)
                        return ops.silu_mul(gu[:, :T * F], gu[:, T * F:])
                    us = timer(dense_gate_up)
                    record(like, "expert_gate_up", us, 4.0 * rows * T * C * F, 2 * C * T * F * 2 + rows * (C + T * F) * 2)
                    mid = rnd(rows, T * F)
                    us = timer(lambda: torch.mm(mid, SL["down"].t()))
                    record(like, "expert_down", us, 2.0 * rows * T * C * F, C * T * F * 2 + rows * (T * F + C) * 2)
                    del act, part, gu, mid
                if want("projection"):
                    us = timer(lambda: torch.addmm(L["bqkv"], h, L["wqkv"].t()))
                    record(ours, "projection_qkv", us, 2.0 * rows * L["wqkv"].numel(), L["wqkv"].numel() * 2 +
                           rows * (C + L["wqkv"].shape[0]) * 2)
                    us = timer(lambda: torch.mm(h, SL["wqkv"].t()))
                    record(like, "projection_qkv", us, 2.0 * rows * SL["wqkv"].numel(), SL["wqkv"].numel() * 2 +
                           rows * (C + SL["wqkv"].shape[0]) * 2)
                out[phase] = {"gifetar": ours, "decoder_stack": like,
                              "distance_ratio": {k: round(ours[k]["times_roofline"] / like[k]["times_roofline"], 2)
                                                 for k in ours if k in like}}
            gif.check_status()
            result["sizes"][size] = out
            del gif, stack, L, SL
            torch.cuda.empty_cache()
    result["gpu_launches"] = ops.launch_count() - launches0
    result["clocks"] = sampler.summary()
    return result
