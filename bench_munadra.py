"""Munadra layers beside Gifetar layers of equal size (`python bench.py --micro munadra`).

Equal size: the same width, heads, feed-forward (experts, top, inner size) and sequence lengths; two layers each, Munadra
with one recurrent and one latent-attention layer.  Random weights, synthetic tokens and caches.  For each size:
throughput of a prompt and of a decode step through Engine's model calls, and each kernel alone -- with its time, its
roofline time (the larger of flops / matrix peak and bytes / copy peak) and how many times longer it takes -- beside the
like kernel of Gifetar: attention and append beside its own, element-wise steps beside the row norms, block-diagonal and
head-wise products beside the projection GEMM.

Kernels are timed with CUDA events on their stream, a write of 256 MB (twice the L2) in front of every call, median of
the calls; the steps without a flush (their weights and caches exceed the L2)."""
from __future__ import annotations

import torch

from bench_gifetar import Timer, _peaks, _step_ms

SIZES = {
    # width, heads, kv heads (Gifetar's), recurrence width and blocks, experts, top, ff | prompt tokens, batch, context
    "w2048": dict(width=2048, heads=16, kv_heads=4, lru=2048, blocks=8, experts=64, top=8, ff=768, prompt=8192, batch=64,
                  ctx=8192),
    "w4096": dict(width=4096, heads=32, kv_heads=8, lru=4096, blocks=16, experts=32, top=4, ff=2048, prompt=8192, batch=128,
                  ctx=4096),
}
VOCAB, DIM, ROT, VDIM, RANK, TAPS, DENSE = 32768, 128, 64, 128, 512, 4, 3
LIKE = {"attention": "attention", "append": "append", "row_norms": "row_norms", "router": "router",
        "experts_gate_up": "experts_gate_up", "experts_down": "experts_down", "projection_latent": "projection",
        "projection_lru": "projection", "expand_latents": "projection", "gather_latents": "append", "query_expansion": "projection",
        "value_expansion": "projection", "lru_gate_products": "projection", "lru_conv": "row_norms", "lru_scan": "row_norms", "lru_step": "row_norms",
        "dense_gate_up": "projection", "dense_activation": "row_norms", "output_projection": "projection"}


def run(args, clock_sampler):
    import kinetics_b200 as kb
    from kinetics_b200 import layer_ops as lo, ops
    from kinetics_b200 import gifetar as gf, munadra as mn

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    hbm, mm, peak_of = _peaks()
    timer = Timer(dev, max(3, min(args.steps, 20)))
    sampler = clock_sampler(0)
    result = {"micro": "munadra", "peaks": {"bytes_per_s": hbm, "flops_per_s": mm, "of": peak_of},
              "l2": "256 MB written in front of every kernel call; steps exceed the L2", "vocab": VOCAB, "sizes": {}}
    launches0 = ops.launch_count()

    with sampler:
        for size, z in SIZES.items():
            C, H, E, T, F = (z[k] for k in ("width", "heads", "experts", "top", "ff"))
            n, B, ctx = z["prompt"], z["batch"], z["ctx"]
            rotation = lo.Rotation(ROT, 1e5, factor=4.0, original=4096, fast=32.0, slow=1.0, scaled=True)
            lat = mn.LatentSpec(H, DIM, ROT, VDIM, RANK, (DIM + ROT) ** -0.5, rotation)
            rec = mn.LruSpec(z["blocks"], z["lru"] // z["blocks"], TAPS)
            mc = mn.MunadraConfig(VOCAB, C, 1e-6, 1.0, 1.0, 30.0, tuple(
                mn.MunadraLayer(s, ff=F, experts=E, top=T, limit=7.0) for s in (rec, lat)))
            layer = gf.GifetarLayer(heads=H, kv_heads=z["kv_heads"], dim=64, vdim=128, scale=0.125, softcap=30.0, diff=0.3,
                                    temp_coef=0.1, temp_every=2048, experts=E, top=T, ff=F)
            gc = gf.GifetarConfig(VOCAB, C, 1e-6, 0.3, (layer,) * 2)
            models = {"munadra": mn.Munadra(mc, mn.random_weights(mc, args.seed, dev), dev),
                      "gifetar": gf.Gifetar(gc, gf.random_weights(gc, args.seed, dev), dev)}
            out = {"config": dict(z, dim=DIM, rot_dim=ROT, vdim=VDIM, rank=RANK)}
            if not args.only_kernel:
                out["steps"] = {name: _steps(kb, m, n, B, ctx, dev) for name, m in models.items()}
            out.update(_kernels(args, models, rec, lat, n, B, ctx, dev, timer, hbm, mm))
            for m in models.values():
                m.check_status()
            result["sizes"][size] = out
            del models
            torch.cuda.empty_cache()
    result["gpu_launches"] = ops.launch_count() - launches0
    result["clocks"] = sampler.summary()
    return result


def _steps(kb, model, n, B, ctx, dev):
    """A prompt of n tokens and a decode step of B sequences behind ctx tokens, ms and tokens per second."""
    tokens, pos = torch.randint(0, VOCAB, (1, n), device=dev), torch.arange(n, device=dev)[None]
    slot0 = torch.tensor([0], device=dev)
    kv = model.new_cache(1, n + 256)

    def prompt():
        kv.clear_cache(0)
        kv.admit(0, n, n)
        kv.begin_step([0])
        model.next_tokens(tokens, pos, slot0, kv, last_only=True)
    ms = _step_ms(prompt, 5)
    kv.check_status()
    del kv
    kv = model.new_cache(B, ctx + 256)
    for t in kv.k_pages + kv.v_pages + kv.states + kv.rings:
        if t is not None:
            t.normal_()
    kv.assume_filled({s: ctx for s in range(B)}, headroom=200)
    eng = kb.Engine(model, kv, ctx + 256, dev, repeat_check=False)
    for s in range(B):
        eng.slots_occupy_status[s] = True
        eng._offsets_host[s] = eng._prompt_host[s] = ctx
    eng.slots_offsets.fill_(ctx)
    eng.slots_tokens.random_(0, VOCAB)
    slots = list(range(B))
    ms_d = _step_ms(lambda: eng.decode_graphed(slots), 30)
    kv.check_status()
    eng._graph = None
    return {"prefill_ms": ms, "prefill_tokens_per_s": n / ms * 1e3, "decode_ms": ms_d, "decode_tokens_per_s": B / ms_d * 1e3}


def _table(lo, batch, length, dev, gen, ps=64):
    pages = (length + ps - 1) // ps
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    perm = torch.randperm(batch * pages, device=dev, generator=gen).to(torch.int32)
    return lo.PageTable(perm, i32([i * pages for i in range(batch + 1)]), i32([length - (pages - 1) * ps] * batch), ps, batch * pages)


def _kernels(args, models, rec, lat, n, B, ctx, dev, timer, hbm, mm):
    from kinetics_b200 import layer_ops as lo
    gen = torch.Generator(device=dev).manual_seed(args.seed)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=gen).to(torch.bfloat16)
    out = {}
    M, G = models["munadra"], models["gifetar"]
    LR, LA, LG = M.layers[0], M.layers[1], G.layers[0]
    C = M.width
    for phase, rows in (("prefill", n), ("decode", B)):
        prompt = phase == "prefill"
        batch, length = (1, n) if prompt else (B, ctx)
        keys = n * (n + 1) / 2 if prompt else batch * length
        indptr = torch.tensor([0, n], dtype=torch.int32, device=dev) if prompt else None
        new = n if prompt else 1
        table = _table(lo, batch, length, dev, gen)
        h, x, y = rnd(rows, C), torch.randn(rows, C, device=dev, generator=gen), rnd(rows, C)
        ours, like = {}, {}

        def record(tab, name, fn, flop=0.0, nbytes=0.0, before=None):
            if args.only_kernel not in name:
                return
            us, roof = timer(fn, before), max(flop / mm, nbytes / hbm) * 1e6
            tab[name] = {"us": round(us, 2), "roofline_us": round(roof, 2), "times_roofline": round(us / roof, 2),
                         "bound": "matrix" if flop / mm > nbytes / hbm else "hbm"}

        def gemm(tab, name, a, w, fn=None):
            record(tab, name, fn or (lambda: torch.mm(a, w.t())), 2.0 * a.shape[0] * w.numel(),
                   2.0 * (w.numel() + a.numel() + a.shape[0] * w.shape[0]))

        # ---- Gifetar
        s = LG["spec"]
        proj = rnd(rows, s.q_cols + s.k_cols + s.v_cols)
        kp, vp = (rnd(batch * ((length + 63) // 64), hd, 64, c) for hd, c in ((s.kv_heads * 2, s.dim_stride), (s.kv_heads, s.vdim_stride)))
        splits = lo.attention_splits(s, batch, length, torch.bfloat16)
        record(like, "attention", lambda: lo.paged_attention(proj, kp, vp, table, s, indptr, new, 1 if prompt else splits),
               keys * s.heads * 4 * (s.dim + s.vdim), batch * length * s.kv_heads * (2 * s.dim + s.vdim) * 2 + rows * (s.q_cols + s.o_cols) * 2)
        record(like, "append", lambda: lo.kv_append(proj, s.q_cols, s.q_cols + s.k_cols, kp, vp, table, s, indptr),
               0, 2 * rows * (s.k_cols + s.v_cols) * 2)
        del kp, vp, proj
        gemm(like, "projection", h, LG["wqkv"], lambda: torch.addmm(LG["bqkv"], h, LG["wqkv"].t()))
        record(like, "row_norms", lambda: lo.residual_norm(x, h, C, 1e-6, pre=LG["norm2"], y=y, post=LG["norm1b"], mult=0.3),
               0, rows * C * 12)

        # ---- latent attention
        w, R, D, H = LA["mix"], lat.rank, lat.row_cols, lat.heads
        pages = rnd(batch * ((length + 63) // 64), 1, 64, D)
        proj = rnd(rows, lat.proj_cols)
        gate = proj[:, lat.gate_col:]
        gemm(ours, "projection_latent", h, LA["proj"])
        q = torch.empty(rows, H, D, dtype=torch.bfloat16, device=dev)
        rotated = 2.0 * rows * H * lat.rot_dim * 2
        record(ours, "append", lambda: lo.latent_append(proj, lat, table, pages, w.norm, w.freqs, indptr, None if prompt else q),
               0, 2 * rows * D * 2 + rotated)
        heads = proj[:, :lat.q_cols].view(rows, H, -1)
        if prompt:
            record(ours, "gather_latents", lambda: lo.gather_rows(pages, table, n), 0, 2.0 * n * D * 2)
            latents = lo.gather_rows(pages, table, n)
            gemm(ours, "expand_latents", latents[:, :R], w.ukv)
            kv = torch.mm(latents[:, :R], w.ukv.t())
            record(ours, "attention", lambda: lo.expanded_attention(proj, kv, latents, lat, w.sink, gate),
                   keys * H * 2 * (DIM + ROT + VDIM), n * H * (DIM + VDIM) * 2 + n * ROT * 2 + rows * H * (DIM + ROT + VDIM) * 2)
            del kv, latents
        else:
            spec = lat.rows()
            splits = lo.attention_splits(spec, batch, length, torch.bfloat16)
            record(ours, "query_expansion", lambda: torch.bmm(heads[:, :, :DIM].transpose(0, 1), w.uk, out=q[:, :, :R].transpose(0, 1)),
                   2.0 * rows * H * DIM * R, 2.0 * (H * DIM * R + rows * H * (DIM + R)))
            q.normal_()
            record(ours, "attention", lambda: lo.paged_attention(q.view(rows, -1), pages, pages, table, spec, None, 1, splits,
                                                                 sink=w.sink, gate=gate),
                   keys * H * 2 * (D + R), batch * length * D * 2 + rows * H * (D + R) * 2)
            o, v = rnd(rows, H, R), rnd(rows, H, VDIM)
            record(ours, "value_expansion", lambda: torch.bmm(o.transpose(0, 1), w.uv.transpose(1, 2), out=v.transpose(0, 1)),
                   2.0 * rows * H * VDIM * R, 2.0 * (H * VDIM * R + rows * H * (VDIM + R)))
        gemm(ours, "output_projection", rnd(rows, H * VDIM), LA["out"])
        del pages, proj, q, heads, gate

        # ---- recurrence
        w, W = LR["mix"], rec.cols
        proj, slots = rnd(rows, 2 * W), torch.arange(batch, dtype=torch.int32, device=dev)
        state, ring = torch.zeros(batch, W, device=dev), torch.zeros(batch, rec.taps, W, dtype=torch.bfloat16, device=dev)
        kw = dict(new_indptr=indptr, max_new=new)
        gemm(ours, "projection_lru", h, LR["proj"], lambda: torch.addmm(LR["proj_b"], h, LR["proj"].t()))
        if prompt:
            record(ours, "lru_conv", lambda: lo.lru_conv(proj, rec, table, slots, w.conv_w, w.conv_b, ring, **kw), 0,
                   rows * W * 4)
            u = rnd(rows, W)
            record(ours, "lru_gate_products", lambda: lo.lru_gate_products(u, w.gates, rec), 4.0 * rows * W * W / rec.blocks,
                   rows * W * (2 + 8) + w.gates.numel() * 2)
            zz = lo.lru_gate_products(u, w.gates, rec)
            record(ours, "lru_scan", lambda: lo.lru_scan(zz, u, proj, rec, table, slots, w.rb, w.ib, w.decay, state, **kw), 0,
                   rows * W * (8 + 2 + 2 + 2))
        else:
            record(ours, "lru_step", lambda: lo.lru_decode(proj, rec, table, slots, w.conv_w, w.conv_b, w.gates, w.rb, w.ib, w.decay,
                                                           ring, state), 4.0 * rows * W * W / rec.blocks,
                   rows * W * (2 * (rec.taps + 1) + 2 + 2 + 8) + w.gates.numel() * 2)
        del proj

        # ---- feed-forward
        record(ours, "row_norms", lambda: lo.residual_norm(x, h, C, 1e-6, y=y, post=LA["norm1"], center=False), 0, rows * C * 12)
        for tab, L in ((ours, LA), (like, LG)):
            _experts(lo, record, tab, L, h, x, rnd, prompt)
        F = DENSE * C
        dense = rnd(2 * F, C)
        gemm(ours, "dense_gate_up", h, dense)
        gu = rnd(rows, 2 * F)
        record(ours, "dense_activation", lambda: lo.gated_rows(gu), 0, rows * F * 6)
        del dense, gu
        ratio = {k: round(v["times_roofline"] / like[LIKE[k]]["times_roofline"], 2) for k, v in ours.items() if LIKE.get(k) in like}
        out[phase] = {"munadra": ours, "gifetar": like, "distance_ratio": ratio}
    return out


def _experts(lo, record, tab, L, h, x, rnd, prompt):
    import ctypes
    from kinetics_b200 import _lib, ops
    moe, (rows, C) = L["moe"], h.shape
    E, T, F = moe.experts, moe.top, moe.ff
    h = h.copy_(x)
    record(tab, "router", lambda: lo.moe_route(h, L["router"], L["router_b"], moe, L["counts"]), 2.0 * rows * E * C,
           rows * C * 2 + E * C * 2 + rows * T * 12, before=lambda: L["counts"].zero_())
    L["counts"].zero_()
    r = lo.moe_route(h, L["router"], L["router_b"], moe, L["counts"])
    used = int((r.counts > 0).sum())
    lib, m = _lib.load_layers(), moe.c(1)
    act, part = rnd(rows * T, F), rnd(rows, T, C)

    def stage(which, src, w, dst):
        _lib.check_layers(lib.ktk_moe_gemm(which, ops._ptr(src), ops._ptr(w), ops._ptr(dst), ops._ptr(r.weights),
                                           ops._ptr(r.counts), ops._ptr(r.bucket), rows, ctypes.byref(m), 0, None, ops._stream()))
    record(tab, "experts_gate_up", lambda: stage(0, h, L["gate_up"], act), 4.0 * rows * T * C * F,
           used * 2 * C * F * 2 + rows * (C + T * F) * 2)
    record(tab, "experts_down", lambda: stage(1, act, L["down"], part), 2.0 * rows * T * C * F,
           used * C * F * 2 + rows * T * (F + C) * 2)
