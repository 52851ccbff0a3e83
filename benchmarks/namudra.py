#!/usr/bin/env python
"""Throughput of the `Namudra` design (llm_decoder.hybrid: a residual of several mixed streams, windowed sigmoid attention
whose values are its keys, latent attention, rotated retention, silu-gated dense layers) at layer sizes that resemble a real
model, next to the framework's closest existing models -- the same config-driven stack serving `Dubarax` (windowed attention
through the same attention kernels, linear attention through the same scan) and `Domilix` (latent attention) -- at equal
width, layer count, vocabulary, batch and context; random weights, synthetic tokens.  `python bench.py --namudra` prints its
JSON line.

Per size: prefill tokens/s (PREFILL_SEQS prompts of PREFILL_LEN tokens in one step) and decode tokens/s (DECODE_SEQS
sequences at DECODE_CTX tokens of context, one token each per step), CUDA events around back-to-back steps after
warm-up.  `kernels` times the design's own kernels alone at the largest size, each next to the like kernel of the other
designs (names ending in `~`), against their roofline (algorithmic bytes over the measured copy bandwidth, FLOPs over the
measured bf16 GEMM rate; MEASURED_PEAKS.json), with L2 flushed before every timed launch."""
import json
import math
import os
import statistics
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PKG = os.path.join(ROOT, "pagedattention-based-transformer-decoder-inference-framework_b200")
for p in (ROOT, PKG):
    if p not in sys.path:
        sys.path.insert(0, p)

from benchmarks import dubarax as du  # noqa: E402
from benchmarks import hybrid as hy  # noqa: E402
from benchmarks import latent as la  # noqa: E402

PREFILL_SEQS, PREFILL_LEN = hy.PREFILL_SEQS, hy.PREFILL_LEN
DECODE_SEQS, DECODE_CTX = hy.DECODE_SEQS, hy.DECODE_CTX
VOCAB = hy.VOCAB
SIZES = {
    "w1024": dict(width=1024, streams=4, heads=8, kv_heads=2, dim=128, window=1024, lat_heads=8, lat_dim=64, rot_dim=32, lat_vdim=64,
                  kv_rank=256, q_rank=384, ret_heads=8, ret_dim=64, ret_vdim=128, ff=2816),
    "w2048": dict(width=2048, streams=4, heads=16, kv_heads=4, dim=128, window=1024, lat_heads=16, lat_dim=128, rot_dim=64,
                  lat_vdim=128, kv_rank=512, q_rank=768, ret_heads=16, ret_dim=64, ret_vdim=128, ff=5632),
}
timed, peaks = hy.timed, hy.peaks


def namudra_config(s):
    dense = {"kind": "dense", "ff": s["ff"]}
    win = {"type": "attention", "mlp": dense,
           "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "mask": {"size": s["window"]},
                     "scale": s["dim"] ** -0.5}}
    lat = {"type": "latent_attention", "mlp": dense,
           "mixer": {"heads": s["lat_heads"], "dim": s["lat_dim"], "rot_dim": s["rot_dim"], "vdim": s["lat_vdim"], "kv_rank": s["kv_rank"],
                     "q_rank": s["q_rank"], "rot": {"dims": s["rot_dim"], "base": 100000.0},
                     "scale": (s["lat_dim"] + s["rot_dim"]) ** -0.5}}
    ret = {"type": "retention", "mlp": None,
           "mixer": {"heads": s["ret_heads"], "dim": s["ret_dim"], "vdim": s["ret_vdim"], "rot": {"dims": s["ret_dim"], "base": 10000.0},
                     "decay": [1.0 - 2.0 ** (-2 - 6 * h / s["ret_heads"]) for h in range(s["ret_heads"])]}}
    return {"architecture": "Namudra", "norm": {"eps": 1e-5}, "vocab": VOCAB, "width": s["width"], "streams": s["streams"],
            "layers": [win, lat, ret, lat], "loop": {"start": 1, "stop": 3, "times": 1}}


def namudra_weights(config, dev):
    g = torch.Generator(device=dev).manual_seed(0)
    Wd, S = config["width"], config["streams"]
    mat = lambda o, i: (torch.randn(o, i, device=dev, generator=g) / math.sqrt(i)).to(torch.bfloat16)  # noqa: E731
    vec = lambda n, std=0.02, mean=0.0: (torch.randn(n, device=dev, generator=g) * std + mean).to(torch.bfloat16)  # noqa: E731
    W = {"embed": torch.randn(config["vocab"], Wd, device=dev, generator=g).to(torch.bfloat16), "head": mat(config["vocab"], Wd),
         "final.norm": vec(Wd)}
    for i, lc in enumerate(config["layers"]):
        p, m, c = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        H, D = c["heads"], c["dim"]
        W[p + "norm1"] = vec(Wd)
        for q in (1, 2) if lc["mlp"] else (1,):
            W[p + f"hc{q}.in"], W[p + f"hc{q}.out"] = vec(S, 0.02, 1.0 / S), vec(S, 0.1, 1.0)
            W[p + f"hc{q}.mix"] = (torch.eye(S, device=dev) * 0.9 + vec(S * S).reshape(S, S).float()).to(torch.bfloat16)
        if lc["type"] == "attention":
            G = c["kv_heads"]
            W[m + "q"], W[m + "k"], W[m + "g"], W[m + "o"] = mat(H * D, Wd), mat(G * D, Wd), mat(H * D, Wd), mat(Wd, H * D)
            W[m + "q.norm"], W[m + "k.norm"], W[m + "pb"] = vec(D, 0.02, 1.0), vec(D, 0.02, 1.0), vec(H, 0.5, -4.0)
        elif lc["type"] == "latent_attention":
            r, V, kr, qr = c["rot_dim"], c["vdim"], c["kv_rank"], c["q_rank"]
            W[m + "dq"], W[m + "dq.norm"], W[m + "uq"] = mat(qr, Wd), vec(qr, 0.02, 1.0), mat(H * (D + r), qr)
            W[m + "dkv"], W[m + "dkv.norm"] = mat(kr + r, Wd), vec(kr, 0.02, 1.0)
            W[m + "uk"], W[m + "uv"], W[m + "o"] = mat(H * D, kr), mat(H * V, kr), mat(Wd, H * V)
        else:
            V = c["vdim"]
            W[m + "q"], W[m + "k"], W[m + "v"] = mat(H * D, Wd), mat(H * D, Wd), mat(H * V, Wd)
            W[m + "g"], W[m + "o"] = mat(H * V, Wd), mat(Wd, H * V)
        if lc["mlp"]:
            ff = lc["mlp"]["ff"]
            W[p + "norm2"] = vec(Wd)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = mat(ff, Wd), mat(ff, Wd), mat(Wd, ff)
    return W


def bench_model(s, dtype, dev):
    import llm_decoder as ld
    config = namudra_config(s)
    cap = DECODE_SEQS * (DECODE_CTX + 64)
    model = ld.HybridDecoder(config, namudra_weights(config, dev), dtype, max_tokens=cap, max_seqs=DECODE_SEQS, tile_size=16)
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


class ColdTimer:
    """Median device time of a call: every timed launch has its own pair of events and finds L2 flushed (a buffer of twice its
    size was written in between)."""

    def __init__(self, dev):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)

    def __call__(self, fn, warmup=3, iters=9):
        for _ in range(warmup):
            fn()
        ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(iters)]
        for a, b in ev:
            self.flush.zero_()
            a.record()
            fn()
            b.record()
        torch.cuda.synchronize()
        return statistics.median(a.elapsed_time(b) for a, b in ev) * 1e-3


def bench_kernels(s, dev, only=None):
    """The design's own kernels alone (bfloat16 activations) at the prefill and decode shapes of size `s`, each followed by
    the like kernel of another design on operands of the same sizes (names ending in `~`)."""
    from llm_decoder import _cabi
    from llm_decoder.hybrid import DECAY_CHUNK, DECAY_CHUNKED_FROM, MMA_FROM, latent_key_splits
    from llm_decoder.seq_state import SequenceStateCache
    lib, st = _cabi.lib(), _cabi.stream
    hbm, tfl, how = peaks()
    cold = ColdTimer(dev)
    out, bf = {}, torch.bfloat16
    W, S, H, G, D = s["width"], s["streams"], s["heads"], s["kv_heads"], s["dim"]

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
        LH, LD, Rt, LV, kvr, qr = s["lat_heads"], s["lat_dim"], s["rot_dim"], s["lat_vdim"], s["kv_rank"], s["q_rank"]
        RH, RD, RV = s["ret_heads"], s["ret_dim"], s["ret_vdim"]
        kd, qd = kvr + Rt, LD + Rt
        states = SequenceStateCache(nseq, nseq * (ctx0 + plen + 16), 16, dev)
        kv = states.add_kv_layer(G, D, 0, "bf16", key_scale=True)
        kv2 = states.add_kv_layer(G, D, D, "bf16")
        kvl = states.add_kv_layer(1, kd, 0, "bf16")
        ret_state = states.add_state(RH * RD * RV)
        slots = [states.alloc() for _ in range(nseq)]
        if ctx0:
            for sl in slots:
                states.extend(sl, ctx0)
        b = states.make_batch([(sl, [1] * plen) for sl in slots])
        for k in (kv, kv2, kvl):
            k.key_buffer_.normal_()
        kv2.value_buffer_.normal_()
        kv.key_scale_.fill_(1.0)
        # ---- windowed attention: sigmoid weights, values = keys, gate; and the other design's window form (bucket table, cap)
        cols = 2 * H * D + G * D
        proj = torch.randn(R, cols, device=dev).to(bf)
        qkv = torch.randn(R, (H + 2 * G) * D, device=dev).to(bf)
        o = torch.empty(R, H * D, device=dev, dtype=bf)
        size = s["window"]
        pb, bucket = torch.randn(H, device=dev) - 4.0, torch.randn(size, H, device=dev)
        tt, mt = lib.pa_masked_attention_tile_tokens(H, G), lib.pa_masked_attention_mma_tile_tokens(D, D, 2)
        pairs = sum(min(i + 1, size) for i in range(plen))
        seen = min(ctx0 + 1, size)
        for kind, group in b.query_tiles(tt, mt, MMA_FROM).items():
            if group is None:
                continue
            tiles, ntiles, _longest = group

            def attend(x, pool, vals, cap, bias, ks, sig, hb, gate_off, kind=3 if kind == 1 else kind):
                pt = pool.page_table_
                return lib.pa_masked_attention_gated(
                    x.data_ptr(), x.stride(0), 0, pool.key_buffer_.data_ptr(), vals.data_ptr(), pt.device_data().data_ptr(), pt.num_beams_,
                    pt.num_heads_, pt.num_tiles_, pool.total_pages_, pool.tile_size_, tiles.data_ptr(), ntiles, H, D, D, D ** -0.5, cap, 1,
                    size, 0, 2 if bias is not None else 0, _cabi.ptr(bias), size if bias is not None else 0, None, None, None, _cabi.ptr(ks),
                    sig, _cabi.ptr(hb), x.data_ptr() if gate_off else None, x.stride(0), gate_off or 0, o.data_ptr(), 2, kind, st())
            mine = lambda: attend(proj, kv, kv.key_buffer_, 0.0, None, kv.key_scale_, 1, pb, H * D + G * D)  # noqa: E731
            other = lambda: attend(qkv, kv2, kv2.value_buffer_, 30.0, bucket, None, 0, None, None)  # noqa: E731
            plain = lambda: attend(qkv, kv2, kv2.value_buffer_, 0.0, None, None, 0, None, None)  # noqa: E731
            if plen > 1:
                rec(f"window_sigmoid_keys_as_values/{tag}", mine, flops=nseq * H * pairs * 4.0 * D)
                rec(f"window_bucket_cap~/{tag}", other, flops=nseq * H * pairs * 4.0 * D)
                rec(f"window_plain_softmax~/{tag}", plain, flops=nseq * H * pairs * 4.0 * D)
            else:
                rec(f"window_sigmoid_keys_as_values/{tag}", mine, bytes_=nseq * seen * G * (D * 2 + 4))
                rec(f"window_bucket_cap~/{tag}", other, bytes_=nseq * seen * G * D * 4)
                rec(f"window_plain_softmax~/{tag}", plain, bytes_=nseq * seen * G * D * 4)
                rec(f"window_sigmoid_keys_as_values streaming/{tag}", lambda: attend(
                    proj, kv, kv.key_buffer_, 0.0, None, kv.key_scale_, 1, pb, H * D + G * D, 1), bytes_=nseq * seen * G * (D * 2 + 4))
                rec(f"window_bucket_cap~ streaming/{tag}", lambda: attend(
                    qkv, kv2, kv2.value_buffer_, 30.0, bucket, None, 0, None, None, 1), bytes_=nseq * seen * G * D * 4)
        gq, gk = torch.ones(D, device=dev), torch.ones(D, device=dev)
        pt, pt2, ptl = kv.page_table_, kv2.page_table_, kvl.page_table_
        rec(f"qk_norm_kv_append/{tag}", lambda: lib.pa_qk_norm_kv_append(
            proj.data_ptr(), cols, 0, H * D, 0, H, G, D, D, gq.data_ptr(), gk.data_ptr(), 1e-5, kv.key_buffer_.data_ptr(), None,
            kv.key_scale_.data_ptr(), pt.device_data().data_ptr(), pt.num_beams_, pt.num_tiles_, kv.total_pages_, kv.tile_size_,
            b.row_slot.data_ptr(), b.row_pos.data_ptr(), R, 2, st()), bytes_=R * (H + G) * D * 4)
        rope_d = torch.empty(R, D // 2, 2, device=dev)
        assert lib.pa_rope_table(b.row_pos.data_ptr(), R, D, 10000.0, rope_d.data_ptr(), st()) == 0
        rec(f"rope_kv_append~/{tag}", lambda: lib.pa_rope_kv_append(
            qkv.data_ptr(), qkv.stride(0), 0, H * D, (H + G) * D, H, G, D, D, D, rope_d.data_ptr(), None, kv2.key_buffer_.data_ptr(),
            kv2.value_buffer_.data_ptr(), pt2.device_data().data_ptr(), pt2.num_beams_, pt2.num_tiles_, kv2.total_pages_, kv2.tile_size_,
            b.row_slot.data_ptr(), b.row_pos.data_ptr(), R, 2, st()), bytes_=R * ((H + 2 * G) * D * 4 + D * 4))
        # ---- retention scan (rotation and key scale inside) and the other design's linear attention; the norm + gate after it
        chunked = plen >= DECAY_CHUNKED_FROM
        items, n, s0, sn = b.chunk_items(DECAY_CHUNK if chunked else 0)
        rc_ = 2 * RH * (RD + RV)
        lin, lo = torch.randn(R, rc_, device=dev).to(bf), torch.empty(R, RH * RV, device=dev)
        decay, rope = torch.full((RH,), 0.97, device=dev), torch.empty(R, RD // 2, 2, device=dev)
        assert lib.pa_rope_table(b.row_pos.data_ptr(), R, RD, 10000.0, rope.data_ptr(), st()) == 0
        wsb = lib.pa_decay_scan_workspace_bytes(n, RH, RD, RV) if chunked else 0
        ws = torch.empty(max(wsb, 16), dtype=torch.uint8, device=dev)

        def scan(act, rp, dims, ksc):
            return lib.pa_decay_scan_rotated(
                lin.data_ptr(), rc_, 0, lin.data_ptr(), rc_, RH * RD, lin.data_ptr(), rc_, 2 * RH * RD, RH, RH, RD, RV, act,
                decay.data_ptr(), None, 0, 0, None, None, None, _cabi.ptr(rp), dims, ksc, ret_state.data_ptr(), lo.data_ptr(), RH * RV,
                items.data_ptr(), n, s0.data_ptr(), sn.data_ptr(), b.seq_slot.data_ptr(), nseq, 1 if chunked else 0, ws.data_ptr(), wsb, 2,
                st())
        io = R * (2 * RH * RD + RH * RV) * 2 + R * RH * RV * 4
        cost = dict(flops=R * RH * RD * RV * 4.0, bytes_=io) if plen > 1 else dict(bytes_=nseq * RH * RD * RV * 8 + io)
        rec(f"retention_scan/{tag}", lambda: scan(0, rope, RD, RD ** -0.5), **cost)
        rec(f"linear_attention_scan~/{tag}", lambda: scan(1, None, 0, 1.0), **cost)
        on, ones = torch.empty(R, RH * RV, device=dev, dtype=bf), torch.ones(RH * RV, device=dev)
        for name, groups, mode, w in (("head_norm_silu_gate", RH, 3, None), ("all_norm_sigmoid_gate~", 1, 2, ones)):
            rec(f"{name}/{tag}", lambda: lib.pa_gated_rms_norm(lo.data_ptr(), R, RH * RV, groups, lin.data_ptr(), rc_, rc_ - RH * RV, mode,
                                                               _cabi.ptr(w), 1e-5, on.data_ptr(), 2, st()), bytes_=R * RH * RV * 8)
        # ---- latent attention: norms + append in one launch (two in the other design), rotation by halves / neighbours, the
        # attention kernel both share, the per-head value product straight into rows / followed by the gate
        lproj = torch.randn(R, qr + kd + LH, device=dev).to(bf)
        gl, gql, cq = torch.ones(kvr, device=dev), torch.ones(qr, device=dev), torch.empty(R, qr, device=dev, dtype=bf)
        rl = torch.empty(R, Rt // 2, 2, device=dev)
        assert lib.pa_rope_table(b.row_pos.data_ptr(), R, Rt, 10000.0, rl.data_ptr(), st()) == 0
        pool = (kvl.key_buffer_.data_ptr(), ptl.device_data().data_ptr(), ptl.num_beams_, ptl.num_tiles_, kvl.total_pages_, kvl.tile_size_)
        rec(f"latent_norm_append/{tag}", lambda: lib.pa_latent_norm_append(
            *pool, kvr, Rt, Rt, 1, lproj.data_ptr(), lproj.stride(0), qr, gl.data_ptr(), 1e-5, rl.data_ptr(), 0, qr, gql.data_ptr(),
            cq.data_ptr(), qr, b.row_slot.data_ptr(), b.row_pos.data_ptr(), R, 2, st()), bytes_=R * (kd + qr) * 4)

        def two_launches():
            lib.pa_rms_norm_rows(lproj.data_ptr(), lproj.stride(0), 0, qr, 1e-5, gql.data_ptr(), cq.data_ptr(), qr, R, 2, st())
            return lib.pa_latent_kv_append(*pool, kvr, Rt, Rt, lproj.data_ptr(), lproj.stride(0), qr, gl.data_ptr(), 1e-5, rl.data_ptr(),
                                           b.row_slot.data_ptr(), b.row_pos.data_ptr(), R, 2, st())
        rec(f"rms_norm_rows+latent_kv_append~/{tag}", two_launches, bytes_=R * (kd + qr) * 4)
        q = torch.randn(R, LH * qd, device=dev).to(bf)
        for name, pairing in (("rope_rows_halves", 1), ("rope_rows_neighbours~", 0)):
            rec(f"{name}/{tag}", lambda: lib.pa_rope_rows_paired(q.data_ptr(), q.stride(0), LD, qd, LH, Rt, rl.data_ptr(), pairing, R, 2,
                                                                 st()), bytes_=R * LH * Rt * 4 + R * Rt * 4)
        w_uk, w_uv = (torch.randn(LH, LD, kvr, device=dev) / math.sqrt(LD)).to(bf), (torch.randn(LH, kvr, LV, device=dev) / math.sqrt(kvr)).to(bf)
        ql = torch.bmm(torch.as_strided(q, (LH, R, LD), (qd, LH * qd, 1)), w_uk)
        latv = torch.randn(LH, R, kvr, device=dev).to(bf)
        tiles, ntiles, longest = b.query_tiles(lib.pa_latent_attention_mma_tile_tokens(LH, kvr, Rt, 2))[1 if plen == 1 else 0]
        nsplit = latent_key_splits(ntiles * math.ceil(LH / 64), longest, _cabi.device_info()[0])
        lwb = lib.pa_latent_attention_workspace_bytes(ntiles, LH, kvr, nsplit)
        lws = torch.empty(max(lwb, 16), dtype=torch.uint8, device=dev)
        keys = plen * (plen + 1) / 2 if plen > 1 else ctx0 + 1
        lcost = dict(flops=nseq * LH * keys * (2.0 * kd + 2 * kvr))
        if plen == 1:
            lcost.update(bytes_=nseq * keys * kd * 2)
        rec(f"latent_attention (shared kernel)/{tag}", lambda: lib.pa_latent_attention(
            ql.data_ptr(), kvr, R * kvr, q.data_ptr() + LD * 2, q.stride(0), qd, *pool, tiles.data_ptr(), ntiles, LH, kvr, Rt, qd ** -0.5,
            latv.data_ptr(), kvr, R * kvr, 2, nsplit, 3 if plen == 1 else 2, lws.data_ptr() if lwb else None, lwb, st()), **lcost)
        ov, og = torch.empty(R, LH, LV, device=dev, dtype=bf), torch.empty(R, LH * LV, device=dev, dtype=bf)
        pcost = dict(flops=2.0 * R * LH * kvr * LV, bytes_=R * LH * (kvr + LV) * 2 + LH * kvr * LV * 2)
        rec(f"value_product_into_rows/{tag}", lambda: torch.bmm(latv, w_uv, out=ov.transpose(0, 1)), **pcost)

        def product_and_gate():
            y = torch.bmm(latv, w_uv)
            return lib.pa_head_gate(y.data_ptr(), LV, R * LV, lproj.data_ptr() + (qr + kd) * 2, lproj.stride(0), LH, LV, R, og.data_ptr(), 2,
                                    st())
        rec(f"value_product+head_gate~/{tag}", product_and_gate, **pcost)
        # ---- the residual streams and the other design's residual step; silu- and relu-gated activations
        x, y, nxt = torch.randn(R, S, W, device=dev), torch.randn(R, W, device=dev).to(bf), torch.empty(R, W, device=dev, dtype=bf)
        mix, vec, g1 = torch.eye(S, device=dev) * 0.9, torch.ones(S, device=dev), torch.ones(W, device=dev)
        rec(f"streams_add_norm/{tag}", lambda: lib.pa_streams_add_norm(
            x.data_ptr(), S, x.data_ptr(), R, S, W, y.data_ptr(), mix.data_ptr(), vec.data_ptr(), vec.data_ptr(), 1e-5, g1.data_ptr(), None,
            nxt.data_ptr(), None, 2, st()), bytes_=R * W * (8 * S + 4))
        x1 = torch.randn(R, W, device=dev)
        rec(f"residual_add_prenorm~/{tag}", lambda: lib.pa_residual_add_prenorm(
            x1.data_ptr(), R, W, y.data_ptr(), 1.0, None, 1.0, None, None, 0, None, None, 1e-5, g1.data_ptr(), nxt.data_ptr(), 2, st()),
            bytes_=R * W * (8 + 4))
        ff = s["ff"]
        gu, a = torch.randn(R, 2 * ff, device=dev).to(bf), torch.empty(R, ff, device=dev, dtype=bf)
        for name, act in (("silu_mul", 0), ("relu_mul~", 1)):
            rec(f"{name}/{tag}", lambda: lib.pa_act_mul(gu.data_ptr(), R, ff, act, a.data_ptr(), 2, st()), bytes_=R * ff * 6)
        del states, kv, kv2, kvl
        torch.cuda.empty_cache()
    out["_denominators"] = dict(hbm_gbs=hbm, bf16_tflops=tfl, source=how)
    return out


def run(sizes=None, kernels=True):
    assert torch.cuda.is_available(), "needs a GPU"
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    res = {"workload": dict(prefill=f"{PREFILL_SEQS} x {PREFILL_LEN} tokens in one step",
                            decode=f"{DECODE_SEQS} sequences at {DECODE_CTX} tokens, one token each per step",
                            layers="windowed sigmoid attention+dense, latent attention+dense, retention, latent attention+dense", vocab=VOCAB,
                            l2="whole steps: inputs larger than L2; kernels: L2 flushed before every timed launch",
                            data="synthetic tokens, random-init weights"), "sizes": {}}
    for name in sizes or SIZES:
        s = SIZES[name]
        res["sizes"][name] = dict(shape=s, namudra_bf16=bench_model(s, "bfloat16", dev), namudra_f32=bench_model(s, "float32", dev),
                                  dubarax_bf16=du.bench_model(du.SIZES[name], "bfloat16", dev),
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
