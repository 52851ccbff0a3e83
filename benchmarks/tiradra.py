#!/usr/bin/env python
"""Throughput of the `Tiradra` design (llm_decoder.hybrid: token-pair embedding, two norms in parallel, causal attention on
convolved, turned and normed projections, latent attention with sinks and an element gate, gelu-gated dense layers) at layer
sizes that resemble a real model, next to the framework's closest existing models -- the same config-driven stack serving
`Gunulorn` (the same wiring, causal attention on convolved projections) and `Domilix` (latent attention) -- at equal width, layer
count, vocabulary, batch and context; random weights, synthetic tokens.  `python bench.py --tiradra` prints its JSON line.

Per size: prefill tokens/s (PREFILL_SEQS prompts of PREFILL_LEN tokens in one step) and decode tokens/s (DECODE_SEQS
sequences at DECODE_CTX tokens of context, one token each per step), CUDA events around back-to-back steps after
warm-up.  `kernels` times the design's own kernels alone at the largest size, each next to the like kernel of the other
designs (names ending in `~`), against their roofline (algorithmic bytes over the measured copy bandwidth, FLOPs over the
measured bf16 GEMM rate; MEASURED_PEAKS.json), with L2 flushed before every timed launch."""
import json
import math
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PKG = os.path.join(ROOT, "pagedattention-based-transformer-decoder-inference-framework_b200")
for p in (ROOT, PKG):
    if p not in sys.path:
        sys.path.insert(0, p)

from benchmarks import gunulorn as gu  # noqa: E402
from benchmarks import hybrid as hy  # noqa: E402
from benchmarks import latent as la  # noqa: E402
from benchmarks.namudra import ColdTimer  # noqa: E402

PREFILL_SEQS, PREFILL_LEN = hy.PREFILL_SEQS, hy.PREFILL_LEN
DECODE_SEQS, DECODE_CTX = hy.DECODE_SEQS, hy.DECODE_CTX
VOCAB = hy.VOCAB
SIZES = {
    "w1024": dict(width=1024, heads=8, kv_heads=2, dim=128, vdim=128, conv=4, lat_heads=8, lat_dim=64, rot_dim=32, lat_vdim=64,
                  kv_rank=256, ff=2816),
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, conv=4, lat_heads=16, lat_dim=128, rot_dim=64, lat_vdim=128,
                  kv_rank=512, ff=5632),
}
timed, peaks = hy.timed, hy.peaks
STRETCH = {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def tiradra_config(s):
    dense = {"kind": "dense", "ff": s["ff"]}
    att = {"type": "attention", "mlp": dense,
           "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "conv": s["conv"],
                     "rot": {"dims": s["dim"], "base": 500000.0, "scaling": STRETCH}, "scale": s["dim"] ** -0.5}}
    lat = {"type": "latent_attention", "mlp": dense,
           "mixer": {"heads": s["lat_heads"], "dim": s["lat_dim"], "rot_dim": s["rot_dim"], "vdim": s["lat_vdim"], "kv_rank": s["kv_rank"],
                     "rot": {"dims": s["rot_dim"], "base": 500000.0, "scaling": STRETCH}, "scale": (s["lat_dim"] + s["rot_dim"]) ** -0.5}}
    return {"architecture": "Tiradra", "norm": {"eps": 1e-5}, "vocab": VOCAB, "width": s["width"], "layers": [att, lat, att, lat],
            "loop": {"start": 1, "stop": 3, "times": 1}, "logit_softcap": 30.0,
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 8191, "mul_cur": 127}}}


def tiradra_weights(config, dev):
    g = torch.Generator(device=dev).manual_seed(0)
    Wd = config["width"]
    mat = lambda o, i: (torch.randn(o, i, device=dev, generator=g) / math.sqrt(i)).to(torch.bfloat16)  # noqa: E731
    vec = lambda n, std=0.02, mean=0.0: (torch.randn(n, device=dev, generator=g) * std + mean).to(torch.bfloat16)  # noqa: E731
    W = {"embed": torch.randn(config["vocab"], Wd, device=dev, generator=g).to(torch.bfloat16), "head": mat(config["vocab"], Wd),
         "bigram": torch.randn(config["embedding"]["bigram"]["buckets"] + 1, Wd, device=dev, generator=g).to(torch.bfloat16),
         "loop.step": vec(config["loop"]["times"] * Wd).reshape(-1, Wd), "final.norm": vec(Wd)}
    for i, lc in enumerate(config["layers"]):
        p, m, c = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        H, D, V = c["heads"], c["dim"], c["vdim"]
        W[p + "norm1"], W[p + "norm2"] = vec(Wd), vec(Wd)
        if lc["type"] == "attention":
            for n, rows in (("q", H * D), ("k", c["kv_heads"] * D), ("v", c["kv_heads"] * V)):
                W[m + n], W[m + n + ".b"] = mat(rows, Wd), vec(rows)
                W[m + n + ".conv"] = (torch.randn(rows, c["conv"], device=dev, generator=g) * 0.5).to(torch.bfloat16)
        else:
            r, kr = c["rot_dim"], c["kv_rank"]
            W[m + "q"], W[m + "dkv"], W[m + "dkv.norm"] = mat(H * (D + r), Wd), mat(kr + r, Wd), vec(kr, 0.02, 1.0)
            W[m + "uk"], W[m + "uv"], W[m + "g"], W[m + "sink"] = mat(H * D, kr), mat(H * V, kr), mat(H * V, Wd), vec(H, 1.0)
        W[m + "o"] = mat(Wd, H * V)
        ff = lc["mlp"]["ff"]
        W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = mat(ff, Wd), mat(ff, Wd), mat(Wd, ff)
    return W


def bench_model(s, dtype, dev):
    import llm_decoder as ld
    config = tiradra_config(s)
    cap = DECODE_SEQS * (DECODE_CTX + 64)
    model = ld.HybridDecoder(config, tiradra_weights(config, dev), dtype, max_tokens=cap, max_seqs=DECODE_SEQS, tile_size=16)
    eng = ld.Engine(model)
    g = torch.Generator().manual_seed(1)
    toks = lambda n: torch.randint(0, VOCAB, (n,), generator=g).tolist()  # noqa: E731
    prompts = [toks(PREFILL_LEN) for _ in range(PREFILL_SEQS)]

    def prefill():
        out = eng.step([(f"p{i}", p, [PREFILL_LEN - 1]) for i, p in enumerate(prompts)])
        for i in range(PREFILL_SEQS):
            eng.finish(f"p{i}")
        return out
    t_pre = timed(prefill, 3, 6)
    for lo in range(0, DECODE_SEQS, 8):
        eng.step([(f"d{i}", toks(DECODE_CTX), []) for i in range(lo, lo + 8)])
    nxt = [toks(1) for _ in range(DECODE_SEQS)]
    t_dec = timed(lambda: eng.step([(f"d{i}", nxt[i], [0]) for i in range(DECODE_SEQS)]), 3, 10)
    for i in range(DECODE_SEQS):
        eng.finish(f"d{i}")
    del model, eng
    torch.cuda.empty_cache()
    return dict(prefill_tok_s=PREFILL_SEQS * PREFILL_LEN / t_pre, prefill_ms=t_pre * 1e3,
                decode_tok_s=DECODE_SEQS / t_dec, decode_ms=t_dec * 1e3)


def bench_kernels(s, dev, only=None):
    """The design's own kernels alone (bfloat16 activations) at the prefill and decode shapes of size `s`, each followed by
    the like kernel of another design on operands of the same sizes (names ending in `~`)."""
    from llm_decoder import _cabi
    from llm_decoder.hybrid import APPEND_CHUNK, CONV_CHUNK, MMA_FROM, latent_key_splits, rotation_scaling, scaled_frequencies
    from llm_decoder.seq_state import SequenceStateCache
    lib, st = _cabi.lib(), _cabi.stream
    hbm, tfl, how = peaks()
    cold = ColdTimer(dev)
    out, bf = {}, torch.bfloat16
    W, H, G, D, V, taps = s["width"], s["heads"], s["kv_heads"], s["dim"], s["vdim"], s["conv"]
    LH, LD, Rt, LV, kvr = s["lat_heads"], s["lat_dim"], s["rot_dim"], s["lat_vdim"], s["kv_rank"]
    kd, qd = kvr + Rt, LD + Rt

    def rec(name, fn, bytes_=None, flops=None):
        if only and not any(name.startswith(o) for o in only):
            return
        rc = fn()
        assert not isinstance(rc, int) or rc == 0, (name, rc)
        secs = cold(fn)
        e = dict(us=secs * 1e6)
        if bytes_ is not None:
            e.update(gbs=bytes_ / secs / 1e9, frac_of_hbm=bytes_ / secs / 1e9 / hbm)
        if flops is not None:
            e.update(tflops=flops / secs / 1e12, frac_of_bf16_gemm=flops / secs / 1e12 / tfl)
        if bytes_ is not None and flops is not None:
            e["frac_of_roofline"] = max(bytes_ / (hbm * 1e9), flops / (tfl * 1e12)) / secs
        out[name] = e

    for tag, nseq, plen, ctx0 in (("prefill", PREFILL_SEQS, PREFILL_LEN, 0), ("decode", DECODE_SEQS, 1, DECODE_CTX)):
        R = nseq * plen
        states = SequenceStateCache(nseq, nseq * (ctx0 + plen + 16), 16, dev)
        states.track_tokens = True
        kv, kvl = states.add_kv_layer(G, D, V, "bf16"), states.add_kv_layer(1, kd, 0, "bf16")
        cols = H * D + G * (D + V)
        conv_state = states.add_state((taps - 1) * cols)
        slots = [states.alloc() for _ in range(nseq)]
        if ctx0:
            for sl in slots:
                states.extend(sl, ctx0)
        b = states.make_batch([(sl, [1] * plen) for sl in slots])
        for k in (kv.key_buffer_, kv.value_buffer_, kvl.key_buffer_):
            k.normal_()
        pt, ptl = kv.page_table_, kvl.page_table_
        table, tablel = pt.device_data(), ptl.device_data()
        # ---- rotation tables: given frequencies, and the plain form
        rope, rl = torch.empty(R, D // 2, 2, device=dev), torch.empty(R, Rt // 2, 2, device=dev)
        freqs, mult = scaled_frequencies(D, 500000.0, rotation_scaling({"scaling": STRETCH}))
        fd = torch.tensor(freqs, dtype=torch.float64, device=dev)
        rec(f"rope_table_scaled/{tag}", lambda: lib.pa_rope_table_scaled(b.row_pos.data_ptr(), R, D, fd.data_ptr(), mult, rope.data_ptr(), st()),
            bytes_=R * D * 4)
        rec(f"rope_table~/{tag}", lambda: lib.pa_rope_table(b.row_pos.data_ptr(), R, D, 500000.0, rope.data_ptr(), st()), bytes_=R * D * 4)
        assert lib.pa_rope_table(b.row_pos.data_ptr(), R, D, 500000.0, rope.data_ptr(), st()) == 0
        assert lib.pa_rope_table(b.row_pos.data_ptr(), R, Rt, 500000.0, rl.data_ptr(), st()) == 0
        # ---- convolution + rotation + norm + append in one launch; the other design's three launches (no norm)
        qkv, q, y = torch.randn(R, cols, device=dev).to(bf), torch.empty(R, H * D, device=dev, dtype=bf), torch.empty(R, cols, device=dev, dtype=bf)
        wt, w = torch.randn(taps, cols, device=dev), torch.randn(cols, taps, device=dev)
        items, n = b.portion_items(APPEND_CHUNK)
        chunks, nch, _a, _b = b.chunk_items(CONV_CHUNK)
        pools = (kv.key_buffer_.data_ptr(), kv.value_buffer_.data_ptr(), table.data_ptr(), pt.num_beams_, pt.num_tiles_, kv.total_pages_, kv.tile_size_)
        io = R * cols * 4 + R * D * 4 + nseq * (taps - 1) * cols * 8
        rec(f"conv_rope_norm_append/{tag}", lambda: lib.pa_conv_rope_norm_append(
            qkv.data_ptr(), cols, 0, H, G, D, V, taps, wt.data_ptr(), conv_state.data_ptr(), D, rope.data_ptr(), 1, 1e-5, q.data_ptr(), H * D,
            *pools, items.data_ptr(), n, APPEND_CHUNK, 2, st()), bytes_=io)

        def three_launches():
            lib.pa_causal_conv(qkv.data_ptr(), cols, 0, cols, taps, w.data_ptr(), None, 0, conv_state.data_ptr(), chunks.data_ptr(), nch,
                               y.data_ptr(), cols, 2, st())
            lib.pa_conv_state_update(qkv.data_ptr(), cols, 0, cols, taps, b.seq_start.data_ptr(), b.seq_len.data_ptr(), b.seq_slot.data_ptr(),
                                     nseq, conv_state.data_ptr(), 2, st())
            return lib.pa_rope_kv_append(y.data_ptr(), cols, 0, H * D, (H + G) * D, H, G, D, V, D, rope.data_ptr(), None, *pools,
                                         b.row_slot.data_ptr(), b.row_pos.data_ptr(), R, 2, st())
        rec(f"causal_conv+conv_state+rope_kv_append~/{tag}", three_launches, bytes_=io)
        # ---- causal attention through the kernel both share; the other design's form (temperature, sink)
        o = torch.empty(R, H * V, device=dev, dtype=bf)
        tt, mt = lib.pa_masked_attention_tile_tokens(H, G), lib.pa_masked_attention_mma_tile_tokens(D, V, 2)
        temp, sink = torch.rand(H, device=dev) + 0.5, torch.randn(max(H, LH), device=dev)
        for kind, group in b.query_tiles(tt, mt, MMA_FROM).items():
            if group is None:
                continue
            tiles, ntiles, _longest = group
            kind = 3 if kind == 1 else kind

            def attend(x, hs, sk):
                return lib.pa_masked_attention_sink(
                    x.data_ptr(), x.stride(0), 0, kv.key_buffer_.data_ptr(), kv.value_buffer_.data_ptr(), table.data_ptr(), pt.num_beams_,
                    pt.num_heads_, pt.num_tiles_, kv.total_pages_, kv.tile_size_, tiles.data_ptr(), ntiles, H, D, V, D ** -0.5, 0.0, 0, 0, 0, 0,
                    None, 0, _cabi.ptr(hs), _cabi.ptr(sk), None, o.data_ptr(), 2, kind, st())
            cost = dict(flops=nseq * H * plen * (plen + 1) * (D + V)) if plen > 1 else dict(bytes_=nseq * (ctx0 + 1) * G * (D + V) * 2)
            rec(f"causal_attention/{tag}", lambda: attend(q, None, None), **cost)
            rec(f"causal_attention_temp_sink~/{tag}", lambda: attend(qkv, temp, sink), **cost)
        # ---- latent attention: append with the queries' rotation / with the query latent's norm; the kernel with and without
        # sinks; the per-head value product with the element gate / the head gate after it
        gcols = LH * LV
        proj = torch.randn(R, LH * qd + kd + gcols, device=dev).to(bf)
        gl = torch.ones(max(kvr, 768), device=dev)
        pool = (kvl.key_buffer_.data_ptr(), tablel.data_ptr(), ptl.num_beams_, ptl.num_tiles_, kvl.total_pages_, kvl.tile_size_)
        rows = (b.row_slot.data_ptr(), b.row_pos.data_ptr(), R, 2, st())
        rec(f"latent_turn_append/{tag}", lambda: lib.pa_latent_turn_append(
            *pool, kvr, Rt, Rt, 0, proj.data_ptr(), proj.stride(0), LH * qd, gl.data_ptr(), 1e-5, rl.data_ptr(), proj.data_ptr(), proj.stride(0), LD,
            LH, qd, *rows), bytes_=R * (kd + LH * Rt) * 4 + R * Rt * 4)

        def append_and_turn():
            lib.pa_latent_kv_append(*pool, kvr, Rt, Rt, proj.data_ptr(), proj.stride(0), LH * qd, gl.data_ptr(), 1e-5, rl.data_ptr(), *rows)
            return lib.pa_rope_rows_paired(proj.data_ptr(), proj.stride(0), LD, qd, LH, Rt, rl.data_ptr(), 0, R, 2, st())
        rec(f"latent_kv_append+rope_rows~/{tag}", append_and_turn, bytes_=R * (kd + LH * Rt) * 4 + R * Rt * 4)
        w_uk, w_uv = (torch.randn(LH, LD, kvr, device=dev) / math.sqrt(LD)).to(bf), (torch.randn(LH, kvr, LV, device=dev) / math.sqrt(kvr)).to(bf)
        ql = torch.bmm(torch.as_strided(proj, (LH, R, LD), (qd, proj.stride(0), 1)), w_uk)
        latv = torch.randn(LH, R, kvr, device=dev).to(bf)
        tiles, ntiles, longest = b.query_tiles(lib.pa_latent_attention_mma_tile_tokens(LH, kvr, Rt, 2))[1 if plen == 1 else 0]
        nsplit = latent_key_splits(ntiles * math.ceil(LH / 64), longest, _cabi.device_info()[0])
        lwb = lib.pa_latent_attention_workspace_bytes(ntiles, LH, kvr, nsplit)
        lws = torch.empty(max(lwb, 16), dtype=torch.uint8, device=dev)
        keys = plen * (plen + 1) / 2 if plen > 1 else ctx0 + 1
        lcost = dict(flops=nseq * LH * keys * (2.0 * kd + 2 * kvr))
        if plen == 1:
            lcost.update(bytes_=nseq * keys * kd * 2)
        for name, sk in (("latent_attention_sink", sink), ("latent_attention~", None)):
            rec(f"{name}/{tag}", lambda: lib.pa_latent_attention_sink(
                ql.data_ptr(), kvr, R * kvr, proj.data_ptr() + LD * 2, proj.stride(0), qd, *pool, tiles.data_ptr(), ntiles, LH, kvr, Rt,
                qd ** -0.5, _cabi.ptr(sk), latv.data_ptr(), kvr, R * kvr, 2, nsplit, 3 if plen == 1 else 2, lws.data_ptr() if lwb else None,
                lwb, st()), **lcost)
        ov, og = torch.empty(R, LH, LV, device=dev, dtype=bf), torch.empty(R, gcols, device=dev, dtype=bf)
        gate = proj.data_ptr() + (LH * qd + kd) * 2
        rec(f"gate_rows/{tag}", lambda: lib.pa_gate_rows(ov.data_ptr(), gcols, gate, proj.stride(0), gcols, R, ov.data_ptr(), gcols, 2, st()),
            bytes_=R * gcols * 6)
        rec(f"head_gate~/{tag}", lambda: lib.pa_head_gate(latv.data_ptr(), LV, R * LV, gate, proj.stride(0), LH, LV, R, og.data_ptr(), 2, st()),
            bytes_=R * gcols * 4)
        pcost = dict(flops=2.0 * R * LH * kvr * LV, bytes_=R * LH * (kvr + LV) * 2 + LH * kvr * LV * 2)

        def product_and_gate():
            torch.bmm(latv, w_uv, out=ov.transpose(0, 1))
            return lib.pa_gate_rows(ov.data_ptr(), gcols, gate, proj.stride(0), gcols, R, ov.data_ptr(), gcols, 2, st())

        def product_and_head_gate():
            v = torch.bmm(latv, w_uv)
            return lib.pa_head_gate(v.data_ptr(), LV, R * LV, gate, proj.stride(0), LH, LV, R, og.data_ptr(), 2, st())
        rec(f"value_product+gate_rows/{tag}", product_and_gate, **pcost)
        rec(f"value_product+head_gate~/{tag}", product_and_head_gate, **pcost)
        # ---- embedding, the residual step, gated activations
        x, x0, step, g1 = torch.randn(R, W, device=dev), torch.randn(R, W, device=dev), torch.randn(W, device=dev), torch.ones(W, device=dev)
        emb, pairs = torch.randn(VOCAB, W, device=dev).to(bf), torch.randn(65522, W, device=dev).to(bf)
        ids = torch.randint(0, VOCAB, (R,), device=dev, dtype=torch.int32)
        rec(f"embedding_bigram/{tag}", lambda: lib.pa_embedding_bigram(emb.data_ptr(), pairs.data_ptr(), 2, ids.data_ptr(), ids.roll(1).data_ptr(), R, W,
                                                                       VOCAB, 65521, 8191, 127, 1.0, x.data_ptr(), x0.data_ptr(), st()),
            bytes_=R * W * 12)
        rec(f"embedding_rows~/{tag}", lambda: lib.pa_embedding_rows_scaled(emb.data_ptr(), 2, ids.data_ptr(), R, W, VOCAB, 1.0, x.data_ptr(), st()),
            bytes_=R * W * 6)
        h, h2, n1, n2 = (torch.randn(R, W, device=dev).to(bf) for _ in range(4))
        for name, base, sv, extra in (("residual_add_norm2_pass", x0, step, 4), ("residual_add_norm2", None, None, 0)):
            rec(f"{name}/{tag}", lambda: lib.pa_residual_add_norm2_pass(
                x.data_ptr(), R, W, h.data_ptr(), h2.data_ptr(), None, None, None, 0, 0, None, _cabi.ptr(base), _cabi.ptr(sv), 1e-5, g1.data_ptr(),
                n1.data_ptr(), g1.data_ptr(), n2.data_ptr(), 2, st()), bytes_=R * W * (16 + extra))
        rec(f"residual_add_prenorm~/{tag}", lambda: lib.pa_residual_add_prenorm(
            x.data_ptr(), R, W, h.data_ptr(), 1.0, None, 1.0, None, None, 0, None, None, 1e-5, g1.data_ptr(), n1.data_ptr(), 2, st()),
            bytes_=R * W * 12)
        ff = s["ff"]
        gu_, a = torch.randn(R, 2 * ff, device=dev).to(bf), torch.empty(R, ff, device=dev, dtype=bf)
        for name, act in (("gelu_tanh_mul", 2), ("silu_mul~", 0), ("relu_mul~", 1)):
            rec(f"{name}/{tag}", lambda: lib.pa_act_mul(gu_.data_ptr(), R, ff, act, a.data_ptr(), 2, st()), bytes_=R * ff * 6)
        del states, kv, kvl
        torch.cuda.empty_cache()
    out["_denominators"] = dict(hbm_gbs=hbm, bf16_tflops=tfl, source=how)
    return out


def run(sizes=None, kernels=True):
    assert torch.cuda.is_available(), "needs a GPU"
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    res = {"workload": dict(prefill=f"{PREFILL_SEQS} x {PREFILL_LEN} tokens in one step",
                            decode=f"{DECODE_SEQS} sequences at {DECODE_CTX} tokens, one token each per step",
                            layers="convolved causal attention+dense, latent attention+dense, convolved causal attention+dense, latent "
                                   "attention+dense", vocab=VOCAB,
                            l2="whole steps: inputs larger than L2; kernels: L2 flushed before every timed launch",
                            data="synthetic tokens, random-init weights"), "sizes": {}}
    for name in sizes or SIZES:
        s = SIZES[name]
        res["sizes"][name] = dict(shape=s, tiradra_bf16=bench_model(s, "bfloat16", dev), tiradra_f32=bench_model(s, "float32", dev),
                                  gunulorn_bf16=gu.bench_model(gu.SIZES[name], "bfloat16", dev),
                                  domilix_bf16=la.bench_model(la.SIZES[name], "bfloat16", dev))
    if kernels:
        res["kernels_w2048_bf16"] = bench_kernels(SIZES["w2048"], dev)
    return res


if __name__ == "__main__":
    if len(sys.argv) >= 3 and sys.argv[1] == "--kernels":     # the kernels alone at one size (a small case for a profiler);
        torch.cuda.set_device(0)                               # further arguments: only kernels whose names start with them
        print(json.dumps({"kernels_" + sys.argv[2]: bench_kernels(SIZES[sys.argv[2]], torch.device("cuda", 0), sys.argv[3:])}, default=float))
    else:
        print(json.dumps(run(), default=float))
