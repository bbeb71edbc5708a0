"""Each hot kernel alone at Llama-4-Scout layer shapes: time (CUDA events, L2 flushed
between iterations), achieved bandwidth or throughput, and the fraction of the measured
peak.  Also the small driver that `ncu` captures for the summaries under `profiles/`.

    python bench_kernels.py                      # all cases, one JSON line each
    python bench_kernels.py --only gemm_decode   # one family (for ncu: -k regex:...)
    python bench_kernels.py --small              # shapes a profiler can replay in seconds
    python bench_kernels.py --only gemm_decode --case "lm_head M=8"   # one case
    python bench_kernels.py --only gemm_decode,moe_decode --rows 4,6   # the decode families at other token counts
    python bench_kernels.py --only attention_decode,attention_prefill --sink 0   # attention with a sink in the softmax
    python bench_kernels.py --only attention_decode,attention_prefill --bias     # ... with a distance bias, learned sinks and gates per head
    python bench_kernels.py --only attention_decode,attention_prefill --latent   # ... over latent rows (one plane, 16 heads on one kv head)
    python bench_kernels.py --only attention_decode,attention_prefill --cap 30             # ... with capped scores
    python bench_kernels.py --only attention_decode,attention_prefill --cap 30 --distance  # ... with a number per head and distance, keys
                                                 # that are the values (one plane) and a factor per key
    python bench_kernels.py --only gated_less    # experts without a gate (squared ReLU), the junction of a loop,
                                                 # the embedding with learned positions
    python bench_kernels.py --only recurrent     # the matrix memory's scan in prompts and decode steps, the heads' norm
    python bench_kernels.py --only scan          # the scans of the state space, the decaying memory and gated linear attention,
                                                 # streams, token shift, gated norm, heads' norm with a silu gate, what is added
                                                 # between two passes, products with silu and gelu gates
    python bench_kernels.py --only delta         # the gated delta rule's scan in prompts and decode steps, the short convolution
                                                 # and gate, the norm behind a sublayer

Families: gemm_decode (weight streaming, mma.sync), gemm_prefill (tcgen05/TMA),
moe_decode, moe_prefill (grouped products), attention_decode, attention_prefill,
small (norm, rotation + cache append, router, sampling), gated_less (what the Sezazen design adds),
recurrent (what the Paposun design adds).
"""
from __future__ import annotations

import argparse
import json
import math
import os
import sys

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)


def main(argv=None):
    import torch
    from bench import peaks
    from spite_b200.cache import LayerCache, Window
    from spite_b200.engine.batch import Segment, build_step_batch
    from spite_b200.kernels.cuda import CudaKernels

    ap = argparse.ArgumentParser()
    ap.add_argument("--only", default="")
    ap.add_argument("--small", action="store_true")
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--case", default="", help="run only the cases whose name contains this text")
    ap.add_argument("--experts", type=int, default=16, help="experts of the grouped products (128: Maverick's)")
    ap.add_argument("--rows", default="1,8,64", help="token counts of the decode families")
    ap.add_argument("--sink", type=float, default=None, help="attention cases run with a sink of this score in the softmax")
    ap.add_argument("--bias", action="store_true", help="attention cases run with a distance bias, a learned sink and a gate per head")
    ap.add_argument("--cap", type=float, default=None, help="attention cases run with scores capped at this")
    ap.add_argument("--wide", action="store_true", help="decode attention in its form of sixteen rows whatever the heads a kv head")
    ap.add_argument("--factors", action="store_true", help="attention cases run on keys that are the values, with a factor per key, alone")
    ap.add_argument("--distance", action="store_true", help="attention cases run with a number per head and distance (32 buckets up to "
                                                          "the context) over keys that are the values, with a factor per key")
    ap.add_argument("--latent", action="store_true", help="attention cases run on a cache of one plane: 16 query heads on one kv head "
                                                        "whose key rows (128 elements) are also the values, the result head by head")
    args = ap.parse_args(argv)
    dev = "cuda:0"
    torch.cuda.set_device(0)
    ks = CudaKernels(torch.bfloat16, dev)
    if args.wide:
        ks.attention_narrow_rows = 0
    pk, src = peaks()
    flush = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device=dev)       # larger than L2
    bf = torch.bfloat16
    d, F, V, nq, nkv, hd, E = 5120, 8192, 202048, 40, 8, 128, args.experts
    if args.small:
        V = 32768
    rnd = lambda *s: (torch.randn(s, device=dev, dtype=torch.float32) * 0.05).to(bf)

    def _timed(fn, iters):
        """One launch between two events, L2 flushed before it.  Includes the launch latency:
        right for kernels of hundreds of microseconds, too pessimistic for short ones."""
        for _ in range(3):
            fn()
        ms = []
        for _ in range(iters):
            flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            ms.append(e0.elapsed_time(e1))
        ms.sort()
        return ms[len(ms) // 2]

    def _timed_rotating(make, nbytes, iters):
        """Short kernels: `make()` builds a launch closure on fresh operands; enough copies are
        made that together they exceed L2 several times, and they run back to back between two
        events, so every launch finds its operands in HBM and no launch gap is counted."""
        n = max(2, min(24, -(-3 * 160 * 1024 * 1024 // max(nbytes, 1))))
        fns = [make() for _ in range(n)]
        for f in fns:
            f()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()              # replayed, so that the host's launch rate does not count
        with torch.cuda.graph(graph):
            for f in fns:
                f()
        best = []
        for _ in range(max(3, iters // 2)):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            graph.replay()
            e1.record()
            torch.cuda.synchronize()
            best.append(e0.elapsed_time(e1) / n)
        best.sort()
        return best[len(best) // 2]

    # the timers are lazy, so that a case filtered out by --case launches nothing
    timed = lambda fn, iters=args.iters: (lambda: _timed(fn, iters))
    timed_rotating = lambda make, nbytes, iters=args.iters: (lambda: _timed_rotating(make, nbytes, iters))

    def report(family, name, timer, nbytes=0, flops=0, **extra):
        if args.case and args.case not in name:
            return
        ms = timer()
        out = {"family": family, "case": name, "us": round(ms * 1e3, 2)}
        if nbytes:
            gbs = nbytes / (ms * 1e-3) / 1e9
            out.update(GBps=round(gbs, 1), hbm_frac=round(gbs / pk["hbm_gbs"], 3))
        if flops:
            tf = flops / (ms * 1e-3) / 1e12
            out.update(TFLOPs=round(tf, 1), bf16_frac=round(tf / pk["bf16_tflops"], 3))
        out.update(peaks=src, **extra)
        print(json.dumps(out), flush=True)

    want = lambda fam: not args.only or fam in args.only.split(",")

    # ---- plain products
    shapes = [("qkv", (nq + 2 * nkv) * hd, d), ("o_proj", d, nq * hd), ("shared_down", d, F), ("lm_head", V, d)]
    decode_rows = tuple(int(m) for m in args.rows.split(","))
    if want("gemm_decode"):
        for M in decode_rows:
            for name, N, K in shapes:
                def make(M=M, N=N, K=K, name=name):
                    x, w = rnd(M, K), rnd(N, K)
                    out = torch.empty((M, N), dtype=torch.float32 if name == "lm_head" else bf, device=dev)
                    return lambda: ks.linear(x, w, out)
                nbytes = 2 * N * K + 2 * M * K + (4 if name == "lm_head" else 2) * M * N
                report("gemm_decode", f"{name} M={M} N={N} K={K}", timed_rotating(make, nbytes), nbytes=nbytes)
            def make(M=M):
                x, w = rnd(M, d), rnd(2 * F, d)
                out = torch.empty((M, F), dtype=bf, device=dev)
                return lambda: ks.linear_swiglu(x, w, out)
            nbytes = 2 * 2 * F * d + 2 * M * d + 2 * M * F
            report("gemm_decode", f"shared_gate_up_swiglu M={M} N=2x{F} K={d}", timed_rotating(make, nbytes),
                   nbytes=nbytes)
    if want("gemm_prefill"):
        for M in ((512,) if args.small else (256, 2048, 8192)):
            for name, N, K in shapes[:3]:
                x, w = rnd(M, K), rnd(N, K)
                out = torch.empty((M, N), dtype=bf, device=dev)
                report("gemm_prefill", f"{name} M={M} N={N} K={K}", timed(lambda: ks.linear(x, w, out)),
                       flops=2 * M * N * K, nbytes=2 * (N * K + M * K + M * N))
                del w
            x, w = rnd(M, d), rnd(2 * F, d)
            out = torch.empty((M, F), dtype=bf, device=dev)
            report("gemm_prefill", f"shared_gate_up_swiglu M={M} N=2x{F} K={d}",
                   timed(lambda: ks.linear_swiglu(x, w, out)), flops=2 * M * 2 * F * d)
            del w
        assert ks.gemm_tc_error() == 0

    # ---- grouped products (experts)
    def routed(M):
        g = torch.Generator(device=dev).manual_seed(M)
        ids = torch.randint(0, E, (M,), device=dev, generator=g)
        order = torch.sort(ids, stable=True)
        offsets = torch.zeros(E + 1, dtype=torch.int32, device=dev)
        offsets[1:] = torch.cumsum(torch.bincount(ids, minlength=E), 0)
        return order.indices.to(torch.int32), offsets, int(ids.unique().numel())
    for fam, Ms in (("moe_decode", decode_rows), ("moe_prefill", (512,) if args.small else (256, 512, 1024, 2048, 8192))):
        if not want(fam):
            continue
        w_gu, w_dn = rnd(E, 2 * F, d), rnd(E, d, F)
        for M in Ms:
            rows, offsets, used = routed(M)
            used = E if M > 64 else used
            x, scale = rnd(M, d), torch.rand(M, device=dev)
            a = torch.empty((M, F), dtype=bf, device=dev)
            h = torch.zeros((M, d), dtype=torch.float32, device=dev)
            report(fam, f"experts_gate_up_swiglu M={M} experts_used={used}",
                   timed(lambda: ks.grouped_linear_swiglu(x, w_gu, rows, offsets, scale, a)),
                   nbytes=used * 2 * 2 * F * d, flops=2 * M * 2 * F * d)
            report(fam, f"experts_down_add M={M} experts_used={used}",
                   timed(lambda: ks.grouped_linear_accumulate(a, w_dn, rows, offsets, h)),
                   nbytes=used * 2 * F * d, flops=2 * M * F * d)
        del w_gu, w_dn

    # ---- what a design without gates in its experts adds: the experts' first product with relu(y)^2 in its epilogue
    # (beside the gated one above: half the weight rows), the junction of a loop, the embedding with learned positions
    if want("gated_less"):
        w_up, w_s = rnd(E, F, d), rnd(F, d)
        for M in decode_rows + ((512,) if args.small else (512, 2048)):
            rows, offsets, used = routed(M)
            used = E if M > 64 else used
            x, scale = rnd(M, d), torch.rand(M, device=dev)
            a = torch.empty((M, F), dtype=bf, device=dev)
            report("gated_less", f"experts_up_relu2 M={M} experts_used={used}",
                   timed(lambda: ks.grouped_linear_act(x, w_up, rows, offsets, scale, a, activation="relu2")),
                   nbytes=used * 2 * F * d, flops=2 * M * F * d)
            report("gated_less", f"shared_up_relu2 M={M} N={F} K={d}",
                   timed(lambda: ks.linear(x, w_s, a, activation="relu2")), nbytes=2 * F * d, flops=2 * M * F * d)
            report("gated_less", f"shared_up_plain_store M={M} N={F} K={d}",
                   timed(lambda: ks.linear(x, w_s, a)), nbytes=2 * F * d, flops=2 * M * F * d)
        del w_up, w_s
        for M in (8, 2048):
            def make_pack(M=M):
                h, h0, step = torch.randn((M, d), device=dev), torch.randn((M, d), device=dev), torch.randn(d, device=dev)
                x = torch.empty((M, 2 * d), dtype=bf, device=dev)
                return lambda: ks.pack_pair(h, h0, x, refill=step)
            report("gated_less", f"pack_pair M={M}", timed_rotating(make_pack, max(M * d * 16, 64 << 20)), nbytes=M * d * 16)
            def make_embed(M=M):
                table, pos_t = rnd(V, d), rnd(8192, d)
                toks = torch.randint(0, V, (M,), dtype=torch.int32, device=dev)
                pos = torch.arange(M, dtype=torch.int32, device=dev)
                h = torch.empty((M, d), dtype=torch.float32, device=dev)
                return lambda: ks.embed(table, toks, h, scale=2.0, position_table=pos_t, positions=pos)
            report("gated_less", f"embed_positions M={M}", timed(make_embed()), nbytes=M * d * 8)

    # ---- attention over the paged cache
    P = 64
    keys_alone = args.distance or args.factors
    one_plane = args.latent or keys_alone
    sink = "" if args.sink is None else f" sink={args.sink}"
    sink += ("" if args.cap is None else f" cap={args.cap}") + (" distance" if args.distance else "") + (" keys as values" if keys_alone else "")
    sink += (" bias+sinks+gates" if args.bias else "") + (" one plane, 16 heads on 1" if args.latent else "")
    if args.latent:
        nq, nkv, hd = 16, 1, 128
    def attention_case(fam, n_req, n_new, ctx, window):
        pages_per = -(-ctx // P)
        win = Window(*window)
        segs, tables, off = [], [], 0
        for r in range(n_req):
            segs.append(Segment(r, r, ctx - n_new, n_new, off, False))
            tables.append(list(range(r * pages_per, (r + 1) * pages_per)))
            off += n_new
        batch = build_step_batch(segs, [[0] * n_new] * n_req, [[]] * n_req, [tables], dev)
        def make():
            kv = (torch.randn((1 if one_plane else 2, n_req * pages_per, nkv, P, hd), device=dev) * 0.5).to(bf)
            q, out = rnd(off, nq * hd), torch.empty((off, nq * hd), dtype=bf, device=dev)
            factors = torch.rand((n_req * pages_per, nkv, P), device=dev) + 0.5 if keys_alone else None
            cache = LayerCache(0, kv, None, P, False, factors)
            more = {} if args.cap is None else {"score_softcap": args.cap}
            if args.distance:
                from spite_b200.kernels.api import DistanceBias
                from spite_b200.parts.position import distance_rows
                more["distance_bias"] = DistanceBias.from_rows(torch.randn((32, nq), device=dev), distance_rows(32, ctx, ctx))
            if args.bias:
                more = {"head_sinks": torch.randn(nq, device=dev), "head_gates": torch.rand((off, nq), device=dev),
                        "head_slopes": torch.tensor([2.0 ** (-8.0 * (h + 1) / nq) for h in range(nq)], device=dev)}
            if args.latent:
                more["out_by_head"] = True
            return lambda: ks.paged_attention(q, out, batch, cache, num_heads=nq, window=win,
                                              softmax_scale=1 / math.sqrt(hd), sink_logit=args.sink, **more)
        seen = sum(min(p + 1, ctx) - win.lowest_visible(p) for p in range(ctx - n_new, ctx)) / n_new
        if n_new == 1:
            # short launches: back to back over rotating copies of the cache, so no launch gap is counted
            nbytes = int(n_req * seen * nkv * (hd * 2 * (1 if one_plane else 2) + (4 if keys_alone else 0)))
            report(fam, f"requests={n_req} context={ctx} window={window[0]}{sink}", timed_rotating(make, nbytes), nbytes=nbytes)
            return
        report(fam, f"tokens={n_new} context={ctx} window={window[0]}{sink}", timed(make()),
               flops=int(n_req * n_new * seen * 4 * nq * hd))
    if want("attention_decode"):
        for n_req in ((8,) if args.small else (1, 8, 64)):
            attention_case("attention_decode", n_req, 1, 2048 if args.small else 8192, ("full", 0))
    if want("attention_prefill"):
        attention_case("attention_prefill", 1, 512 if args.small else 2048, 512 if args.small else 2048, ("full", 0))
        if not args.small:
            attention_case("attention_prefill", 1, 2048, 8192, ("chunk", 8192))
            attention_case("attention_prefill", 1, 8192, 131072, ("full", 0))     # a late portion of a long prompt

    # ---- rotation + per-head norm + cache append, at decode and at prompt lengths
    if want("small"):
        from spite_b200.parts import QkNorm, Rotation
        for M in (8, 2048):
            pages_per = -(-M // P) + 1
            segs = [Segment(0, 0, 0, M, 0, True)]
            batch = build_step_batch(segs, [[0] * M], [[]], [[list(range(pages_per))]], dev)
            inv_freq = torch.tensor([500000.0 ** (-2.0 * i / hd) for i in range(hd // 2)], dtype=torch.float32, device=dev)
            def make_prepare(M=M, batch=batch, pages_per=pages_per):
                qkv = rnd(M, (nq + 2 * nkv) * hd)
                q = torch.empty((M, nq * hd), dtype=bf, device=dev)
                kv = torch.zeros((2, pages_per, nkv, P, hd), dtype=bf, device=dev)
                cache = LayerCache(0, kv, None, P, True)
                return lambda: ks.qk_prepare(qkv, q, batch, cache, num_heads=nq, rotation=Rotation(inv_freq, "neighbours"),
                                             qk_norm=QkNorm(1e-5), temperature=None)
            nbytes = M * ((nq + 2 * nkv) * hd * 2 + (nq + 2 * nkv) * hd * 2)
            report("small", f"qk_prepare M={M}", timed_rotating(make_prepare, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)

    # ---- the kernels between the products of an attention through latents (q_rank 1024, rows of 96 + 32, 16 heads of 64 + 32)
    if want("latent"):
        from spite_b200.parts import Rotation
        rq, rkv, dr, lh, dn, row = 1024, 96, 32, 16, 64, 128
        rot = Rotation(torch.tensor([10000.0 ** (-2.0 * i / dr) for i in range(dr // 2)], dtype=torch.float32, device=dev), "neighbours", dr, 1.1)
        for M in (8, 2048):
            pages_per = -(-M // P) + 1
            batch = build_step_batch([Segment(0, 0, 0, M, 0, True)], [[0] * M], [[]], [[list(range(pages_per))]], dev)
            def make_prepare(M=M, batch=batch, pages_per=pages_per):
                down = torch.randn((M, rq + rkv + dr + lh), device=dev)
                cq, gates = torch.empty((M, rq), dtype=bf, device=dev), torch.empty((M, lh), dtype=torch.float32, device=dev)
                cache = LayerCache(0, torch.zeros((1, pages_per, 1, P, row), dtype=bf, device=dev), None, P, True)
                qg, kg = torch.ones(rq, device=dev), torch.ones(rkv, device=dev)
                return lambda: ks.latent_prepare(down, cq, batch, cache, q_rank=rq, kv_rank=rkv, rotation=rot, q_gain=qg, kv_gain=kg,
                                                 eps=1e-5, num_gates=lh, gates_out=gates)
            nbytes = M * ((rq + rkv + dr + lh) * 4 + rq * 2 + row * 2 + lh * 4)
            report("latent", f"latent_prepare M={M}", timed_rotating(make_prepare, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)
            def make_queries(M=M, batch=batch):
                q, qa = rnd(M, lh * (dn + dr)), torch.empty((M, lh * row), dtype=bf, device=dev)
                qs = torch.empty((lh * M, dn), dtype=bf, device=dev)
                rows, offs = torch.empty(lh * M, dtype=torch.int32, device=dev), torch.empty(lh + 1, dtype=torch.int32, device=dev)
                return lambda: ks.latent_queries(q, qa, batch, num_heads=lh, head_dim=dn, kv_rank=rkv, rotation=rot, rows_out=rows,
                                                 offsets_out=offs, sorted_out=qs)
            nbytes = M * lh * ((dn + dr) * 2 + (row - rkv) * 2 + dn * 2 + 4)
            report("latent", f"latent_queries M={M}", timed_rotating(make_queries, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)

    # ---- the matrix memory's scan (8 heads of 256 key rows and 512 value columns, float32), the heads' norm with gain and
    # gate behind it, and the norm that stands behind a sublayer
    if want("recurrent"):
        H, kd, vd, dm = (8, 128, 256, 2048) if args.small else (8, 256, 512, 4096)
        size = ks.mlstm_state_size(kd, vd)
        cols = (0, H * kd, 2 * H * kd, 2 * H * kd + 2 * H * vd, 2 * H * kd + 2 * H * vd + H)
        width = -(-(cols[4] + H) // 8) * 8
        fma_peak = 148 * 128 * 2 * pk.get("sm_max_mhz", 1965.0) * 1e6            # float32 multiply-adds of the CUDA cores, FLOP/s
        zero = torch.zeros(H, device=dev)
        for n_seg, n_tok in ((1, 2048), (8, 2048), (1, 1), (8, 1), (64, 1)):
            M = n_seg * n_tok
            segs = [Segment(i, i, 0, n_tok, i * n_tok, True) for i in range(n_seg)]
            batch = build_step_batch(segs, [[0] * n_tok] * n_seg, [[]] * n_seg, [[[0]] * n_seg], dev)
            def make_scan(M=M, batch=batch, n_seg=n_seg, chunked=False):
                proj = torch.randn((M, width), device=dev)
                out = torch.empty((M, H * vd), device=dev)
                state = torch.zeros((n_seg, H, size), device=dev)
                return lambda: ks.mlstm_scan(proj, out, batch, state, heads=H, dim=kd, vdim=vd, gate_cap=10.0, q_scale=kd ** -0.5,
                                             columns=cols, i_bias=zero, f_bias=zero, chunked=chunked)
            nbytes = n_seg * H * size * 4 * 2 + M * (2 * H * kd + 2 * H * vd + 2 * H) * 4
            flops = 4 * M * H * kd * vd
            name = f"mlstm_scan {n_seg} x {n_tok} tokens, {H} heads of {kd} x {vd}"
            if n_tok > 1:
                for chunked in (False, True):
                    full = name + (", 32 tokens at a time" if chunked else ", token by token")
                    if args.case and args.case not in full:
                        continue
                    ms = timed(make_scan(chunked=chunked))()
                    print(json.dumps({"family": "recurrent", "case": full, "us": round(ms * 1e3, 2), "TFLOPs_fp32": round(flops / ms / 1e9, 2),
                                      "fp32_fma_frac": round(flops / (ms * 1e-3) / fma_peak, 3), "GBps": round(nbytes / ms / 1e6, 1),
                                      "peaks": src}), flush=True)
            else:
                report("recurrent", name, timed_rotating(make_scan, nbytes), nbytes=nbytes)
        for M in (8, 2048):
            def make_heads(M=M):
                o, proj = torch.randn((M, H * vd), device=dev), torch.randn((M, width), device=dev)
                a, gain = torch.empty((M, H * vd), dtype=bf, device=dev), torch.ones(H * vd, device=dev)
                return lambda: ks.head_norm_gate(o, a, heads=H, size=vd, gates=proj, gate_column=cols[2] + H * vd, gain=gain, eps=1e-6)
            nbytes = M * H * vd * (4 + 4 + 2)
            report("recurrent", f"head_norm_gate M={M}, {H} heads of {vd}", timed_rotating(make_heads, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)
            def make_join(M=M):
                y, h, g1, g2 = torch.randn((M, dm), device=dev), torch.randn((M, dm), device=dev), torch.ones(dm, device=dev), torch.ones(dm, device=dev)
                x = torch.empty((M, dm), dtype=bf, device=dev)
                return lambda: ks.rms_norm_residual(y, g1, 1e-5, 0.5, h, next_gain=g2, next_out=x)
            nbytes = M * dm * (4 + 4 + 4 + 2)
            report("recurrent", f"rms_norm_residual with the next norm M={M} d={dm}", timed_rotating(make_join, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)

    # ---- the gated delta rule's scan (heads of 128 x 128 on half as many q/k heads, float32), the convolution over time in
    # front of it and the cast that a sublayer without a norm in front reads
    if want("delta"):
        dm = 2048 if args.small else 4096
        H, G, kd, vd = dm // 128, dm // 256, 128, 128
        ch = 2 * G * kd + H * vd
        cols = (0, G * kd, 2 * G * kd, ch + H * vd, ch + H * vd + H)
        width = -(-(cols[4] + H) // 8) * 8
        fma_peak = 148 * 128 * 2 * pk.get("sm_max_mhz", 1965.0) * 1e6
        zero = torch.zeros(H, device=dev)
        for n_seg, n_tok in ((1, 2048), (8, 2048), (1, 1), (8, 1), (64, 1)):
            M = n_seg * n_tok
            segs = [Segment(i, i, 0, n_tok, i * n_tok, True) for i in range(n_seg)]
            batch = build_step_batch(segs, [[0] * n_tok] * n_seg, [[]] * n_seg, [[[0]] * n_seg], dev)
            def make_scan(M=M, batch=batch, n_seg=n_seg, split=None):
                x = torch.randn((M, width), device=dev)
                out = torch.empty((M, H * vd), device=dev)
                state = torch.zeros((n_seg, H * kd * vd), device=dev)
                return lambda: ks.delta_scan(x, out, batch, state, heads=H, kv_heads=G, dim=kd, vdim=vd, columns=cols, a_log=zero - 2.0,
                                             dt_bias=zero, q_scale=kd ** -0.5, split_rows=split)
            nbytes = n_seg * H * kd * vd * 4 * 2 + M * (2 * G * kd + 2 * H * vd + 2 * H) * 4
            flops = 4 * M * H * kd * vd
            name = f"delta_scan {n_seg} x {n_tok} tokens, {H} heads of {kd} x {vd}"
            if n_tok > 1:
                for split in (False, True):
                    full = name + (", rows split further" if split else ", eight columns a warp")
                    if args.case and args.case not in full:
                        continue
                    ms = timed(make_scan(split=split))()
                    print(json.dumps({"family": "delta", "case": full, "us": round(ms * 1e3, 2), "TFLOPs_fp32": round(flops / ms / 1e9, 2),
                                      "fp32_fma_frac": round(flops / (ms * 1e-3) / fma_peak, 3), "GBps": round(nbytes / ms / 1e6, 1),
                                      "peaks": src}), flush=True)
            else:
                report("delta", name, timed_rotating(make_scan, nbytes), nbytes=nbytes)
            def make_conv(M=M, batch=batch, n_seg=n_seg):
                x, w = torch.randn((M, width), device=dev), torch.randn((ch, 4), device=dev)
                out = torch.empty((M, width), device=dev)
                state = torch.zeros((n_seg, 3 * ch), device=dev)
                return lambda: ks.short_conv(x, w, out, batch, state, channels=ch, activation="silu")
            nbytes = M * width * 8 + n_seg * 3 * ch * 8
            report("delta", f"short_conv {n_seg} x {n_tok} tokens, {ch} channels of 4 taps", timed_rotating(make_conv, max(nbytes, 64 << 20) if n_tok == 1 else nbytes), nbytes=nbytes)
        for M in (8, 2048):
            def make_cast(M=M):
                h, x = torch.randn((M, dm), device=dev), torch.empty((M, dm), dtype=bf, device=dev)
                return lambda: ks.cast_rows(h, x)
            nbytes = M * dm * 6
            report("delta", f"cast_rows M={M} d={dm}", timed_rotating(make_cast, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)

    # ---- the scans of the state space and of the decaying memory, and what stands around them
    if want("scan"):
        dm = 2048 if args.small else 4096
        fma_peak = 148 * 128 * 2 * pk.get("sm_max_mhz", 1965.0) * 1e6
        for n_seg, n_tok in ((1, 2048), (8, 2048), (1, 1), (8, 1), (64, 1)):
            M = n_seg * n_tok
            segs = [Segment(i, i, 0, n_tok, i * n_tok, True) for i in range(n_seg)]
            batch = build_step_batch(segs, [[0] * n_tok] * n_seg, [[]] * n_seg, [[[0]] * n_seg], dev)
            for kind, H, kd, vd in (("state_space", dm // 32, 128, 64), ("decay", dm // 64, 64, 64), ("gated_linear", dm // 64, 64, 64),
                                    ("gated_linear", dm // 128, 64, 128)):
                G = 1 if kind == "state_space" else H
                size = H * ks.scan_state_size(kd, vd)
                def make_scan(M=M, batch=batch, n_seg=n_seg, kind=kind, H=H, kd=kd, vd=vd, G=G, size=size):
                    out, state = torch.empty((M, H * vd), device=dev), torch.zeros((n_seg, size), device=dev)
                    hv = torch.zeros(H, device=dev)
                    if kind == "state_space":
                        x, step = torch.randn((M, 2 * kd + H * vd), device=dev), torch.randn((M, H), device=dev)
                        return lambda: ks.state_space_scan((x, kd), (x, 0), (x, 2 * kd), (step, 0), out, batch, state, heads=H, kv_heads=1,
                                                           dim=kd, vdim=vd, a_log=hv, dt_bias=hv, skip=hv)
                    if kind == "gated_linear":
                        x, w = torch.randn((M, H * (2 * kd + vd) + 16), device=dev), torch.empty((M, H * kd), device=dev)
                        a2, b = torch.randn((16, H * kd), device=dev), torch.zeros(H * kd, device=dev)
                        return lambda: ks.gated_linear_scan((x, 0), (x, H * kd), (x, 2 * H * kd), (x, H * (2 * kd + vd)), w, out, batch, state,
                                                            heads=H, dim=kd, vdim=vd, a2=a2, a2_bias=b, tau=16.0, q_scale=0.125)
                    r, k, v, w = (torch.randn((M, H * kd), device=dev) for _ in range(4))
                    u = torch.zeros(H * kd, device=dev)
                    return lambda: ks.decay_scan((r, 0), (k, 0), (v, 0), w, out, batch, state, heads=H, dim=kd,
                                                 vdim=vd, w0=u, u=u)
                nbytes = n_seg * size * 8 + M * ((2 * G * kd + 2 * H * vd + H) * 4 + (0 if kind == "state_space" else H * kd * 4))
                flops = 4 * M * H * kd * vd
                name = f"{kind}_scan {n_seg} x {n_tok} tokens, {H} heads of {kd} x {vd}"
                if args.case and args.case not in name:
                    continue
                if n_tok > 1:
                    ms = timed(make_scan())()
                    print(json.dumps({"family": "scan", "case": name, "us": round(ms * 1e3, 2), "TFLOPs_fp32": round(flops / ms / 1e9, 2),
                                      "fp32_fma_frac": round(flops / (ms * 1e-3) / fma_peak, 3), "GBps": round(nbytes / ms / 1e6, 1),
                                      "peaks": src}), flush=True)
                else:
                    report("scan", name, timed_rotating(make_scan, nbytes), nbytes=nbytes)
            inner = 2 * dm
            ch, width = inner + 256, 2 * inner + 256 + dm // 32
            def make_conv(M=M, batch=batch, n_seg=n_seg):
                x, w, b = torch.randn((M, width), device=dev), torch.randn((ch, 4), device=dev), torch.randn(ch, device=dev)
                out, state = torch.empty((M, ch), device=dev), torch.zeros((n_seg, 3 * ch), device=dev)
                return lambda: ks.short_conv(x, w, out, batch, state, channels=ch, activation="silu", bias=b)
            nbytes = M * ch * 8 + n_seg * 3 * ch * 8
            report("scan", f"short_conv with a bias {n_seg} x {n_tok} tokens, {ch} channels of 4 taps", timed_rotating(make_conv, max(nbytes, 64 << 20) if n_tok == 1 else nbytes), nbytes=nbytes)
            def make_shift(M=M, batch=batch, n_seg=n_seg):
                x, mu = rnd(M, dm), torch.rand((5, dm), device=dev)
                out, state = torch.empty((5, M, dm), dtype=bf, device=dev), torch.zeros((n_seg, dm), device=dev)
                return lambda: ks.token_shift(x, mu, out, batch, state)
            nbytes = M * dm * 12 + n_seg * dm * 8
            report("scan", f"token_shift {n_seg} x {n_tok} tokens, 5 mixes of {dm}", timed_rotating(make_shift, max(nbytes, 64 << 20) if n_tok == 1 else nbytes), nbytes=nbytes)
        for M in (8, 2048):
            def make_heads(M=M):
                o, z, g = torch.randn((M, dm), device=dev), torch.randn((M, 2 * dm), device=dev), torch.ones(128, device=dev)
                a = torch.empty((M, dm), dtype=bf, device=dev)
                return lambda: ks.head_norm_gate(o, a, heads=dm // 128, size=128, gates=z, gate_column=dm, gain=g, eps=1e-6, gate_activation="silu")
            nbytes = M * dm * 10
            report("scan", f"head_norm_gate M={M}, {dm // 128} heads of 128, silu gate", timed_rotating(make_heads, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)
            def make_add(M=M):
                h, h0, step = torch.randn((M, dm), device=dev), torch.randn((M, dm), device=dev), torch.randn(dm, device=dev)
                return lambda: ks.fill_rows(h, step, accumulate=True, other=h0)
            nbytes = M * dm * 12
            report("scan", f"fill_rows M={M} d={dm}, two rows and a vector", timed_rotating(make_add, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)
            for act in ("silu", "gelu_tanh"):
                def make_gated(M=M, act=act):
                    x, w, a = rnd(M, dm), rnd(2 * 14336, dm), torch.empty((M, 14336), dtype=bf, device=dev)
                    return lambda: ks.linear_swiglu(x, w, a, activation=act)
                name, flops, nbytes = f"gate and up, {act}, M={M}, 2 x 14336 x {dm}", 4 * M * 14336 * dm, 4 * 14336 * dm
                if M == 8:
                    report("scan", name, timed_rotating(make_gated, nbytes), nbytes=nbytes)
                elif not args.case or args.case in name:
                    report("scan", name, timed(make_gated()), flops=flops)
            inner = 2 * dm
            def make_norm(M=M):
                y, z, g = torch.randn((M, inner), device=dev), torch.randn((M, inner), device=dev), torch.ones(inner, device=dev)
                a = torch.empty((M, inner), dtype=bf, device=dev)
                return lambda: ks.gate_group_norm(y, z, g, a, groups=1, eps=1e-6)
            nbytes = M * inner * 10
            report("scan", f"gate_group_norm M={M}, one part of {inner}", timed_rotating(make_norm, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)
            def make_streams(M=M):
                S = 4
                x, y = torch.randn((M, S, dm), device=dev), torch.randn((M, dm), device=dev)
                mix, wo, wi = torch.eye(S, device=dev).contiguous(), torch.zeros(S, device=dev), torch.ones(S, device=dev)
                sc, b, g = torch.ones(dm, device=dev), torch.zeros(dm, device=dev), torch.ones(dm, device=dev)
                a = torch.empty((M, dm), dtype=bf, device=dev)
                return lambda: ks.streams(x, y=y, bias=b, scale=sc, mix=mix, w_out=wo, w_in=wi, gain=g, eps=1e-6, next_out=a)
            nbytes = M * dm * (4 * 8 + 4 + 2)
            report("scan", f"streams M={M}, four of {dm}, output laid in and next norm", timed_rotating(make_streams, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)
            segs = [Segment(0, 0, 0, M, 0, True)]
            batch = build_step_batch(segs, [[0] * M], [[]], [[[0]]], dev)
            from spite_b200.parts import Rotation
            vrot = Rotation(torch.tensor([500000.0 ** (-2.0 * i / 128) for i in range(64)], dtype=torch.float32, device=dev), "halves", 128)
            def make_turn(M=M, batch=batch):
                h = dm // 128
                x, o = rnd(M, dm), torch.empty((M, 2 * dm), dtype=bf, device=dev)
                return lambda: ks.turn_heads(x, o, batch, heads=h, size=128, rotation=vrot, scale=0.5)
            nbytes = M * dm * 4
            report("scan", f"turn_heads M={M}, {dm // 128} heads of 128", timed_rotating(make_turn, max(nbytes, 64 << 20) if M == 8 else nbytes), nbytes=nbytes)

    # ---- the small kernels of a decode step
    if want("small"):
        for M in (8, 64):
            def make_norm(M=M):
                h, gain = torch.randn((M, d), device=dev), torch.ones(d, device=dev)
                x = torch.empty((M, d), dtype=bf, device=dev)
                return lambda: ks.rms_norm(h, gain, 1e-5, x)
            report("small", f"rms_norm M={M}", timed_rotating(make_norm, 64 << 20), nbytes=M * d * 6)
            def make_route(M=M):
                x, wr = rnd(M, d), torch.randn((E, d), device=dev) * 0.05
                return lambda: ks.moe_route(x, wr, 1)
            report("small", f"router M={M}", timed_rotating(make_route, 64 << 20), nbytes=E * d * 4 + M * d * 2)
            def make_argmax(M=M):
                logits = torch.randn((M, V), device=dev)
                return lambda: ks.argmax(logits)
            report("small", f"argmax M={M} V={V}", timed_rotating(make_argmax, M * V * 4), nbytes=M * V * 4)
            def make_sample(M=M):
                logits = torch.randn((M, V), device=dev) * 3
                f32 = lambda v: torch.full((M,), v, dtype=torch.float32, device=dev)
                ctxt = torch.randint(0, V, (M * 64,), dtype=torch.int32, device=dev)
                offs = torch.arange(0, M * 64 + 1, 64, dtype=torch.int32, device=dev)
                state = torch.arange(M, dtype=torch.int64, device=dev)
                return lambda: ks.sample(logits, temperature=f32(0.7), top_k=torch.zeros(M, dtype=torch.int32, device=dev),
                                         top_p=f32(0.95), min_p=f32(0.0), repetition_penalty=f32(1.1), context=ctxt,
                                         context_offsets=offs, rng_state=state)
            report("small", f"sample (temperature 0.7, top-p 0.95, penalty 1.1) M={M} V={V}",
                   timed_rotating(make_sample, M * V * 4), nbytes=M * V * 4)
    return 0


if __name__ == "__main__":
    sys.exit(main())
