"""The `Namudra` design in the config-driven stack (llm_decoder.hybrid: a residual of several mixed streams, a looped
block, windowed sigmoid attention whose values are its keys, latent attention with a half-pair rotation, rotated
retention; csrc/masked_attention.cu, latent_attention.cu, recurrence_ops.cu, seq_ops.cu) against the plain float64 oracle
(oracle/namudra_ref.py), on small random models of its own making.

The engine's logits at a position must equal the oracle's full recomputation whatever the cut into steps, the batch
around it, and the pages / slots in use."""
import json
import math
import os
import random
import subprocess

import pytest
import torch

from oracle import namudra_ref as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 5e-4      # max abs error of float32 logits (magnitude of a few units)
BF16_TOL = 0.06     # relative rms error of bfloat16 logits, median of the positions


def _model(config, weights, dtype="float32", max_tokens=1024, max_seqs=4, tile_size=16):
    import llm_decoder as ld
    return ld.HybridDecoder(config, weights, dtype, max_tokens=max_tokens, max_seqs=max_seqs, tile_size=tile_size)


def _tokens(n, vocab, seed):
    rnd = random.Random(seed)
    return [rnd.randrange(vocab) for _ in range(n)]


_ORACLE = {}


def _oracle(key, config, weights, tokens):
    k = (key, tuple(tokens))
    if k not in _ORACLE:
        _ORACLE[k] = R.forward(config, weights, tokens)
    return _ORACLE[k]


def _close(got, want, dtype="float32", tol=F32_TOL, bf16_tol=BF16_TOL):
    got, want = got.double().cpu(), want.double()
    if dtype == "float32":
        err = (got - want).abs().max().item()
        assert err < tol * max(1.0, want.abs().max().item() / 4), f"max abs error {err}"
    else:
        got, want = got.reshape(-1, got.shape[-1]), want.reshape(-1, want.shape[-1])
        rel = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
        # the median position carries the bound: where a head of a retention layer is nearly empty, its norm multiplies the
        # rounding of a position many times (float32 carries the exact comparison)
        mid, worst = rel.median().item(), rel.max().item()
        assert math.isfinite(worst) and mid < bf16_tol and worst < 6 * bf16_tol, f"relative rms error {mid} (median), {worst} (worst)"


def _feed(engine, rid, tokens, cuts):
    """Feed `tokens` of one request in portions ending at `cuts`; returns logits of ALL positions."""
    outs, lo = [], 0
    for hi in list(cuts) + [len(tokens)]:
        if hi > lo:
            outs.append(engine.step([(rid, tokens[lo:hi], list(range(hi - lo)))]))
            lo = hi
    return torch.cat(outs, 0)


# ---- configurations: sizes and constants unlike each other -- one to five streams, one, two and three key/value heads, head
# sizes that are no multiples of 8 or 32, windows that are no multiples of a page or a key step, rotation over a part and
# over all of a head, rot_dim above and below dim, vdim above and below dim, loops of one and several layers, of every kind
# of layer, none, and one pass -----------------------------------------------------------------------------------------
def cfg_window():
    return R.make_config([R.window_layer(heads=4, kv_heads=2, dim=16, size=11)], width=64, streams=2)


def cfg_latent():
    return R.make_config([R.latent_layer(heads=3, dim=8, rot_dim=16, vdim=20, q_rank=24, kv_rank=40, base=500.0)], width=64, streams=1)


def cfg_retention():
    return R.make_config([R.retention_layer(heads=3, dim=16, vdim=24, rot_dims=10, base=700.0)], width=64, streams=2)


def cfg_loop():
    return R.make_config([R.retention_layer(heads=2, dim=8, vdim=16, rot_dims=8, ff=40), R.window_layer(heads=2, kv_heads=1, dim=24, size=7, ff=None),
                          R.latent_layer(heads=2, dim=8, rot_dim=8, vdim=8, q_rank=16, kv_rank=16, ff=None)],
                         width=48, streams=4, loop={"start": 0, "stop": 3, "times": 2})


def cfg_full():
    layers = [R.retention_layer(heads=4, dim=24, vdim=16, rot_dims=24, base=300.0, decay=[1.0, 0.9, 0.5, 0.995]),
              R.latent_layer(heads=5, dim=24, rot_dim=8, vdim=40, q_rank=32, kv_rank=72, base=10000.0, ff=72),
              R.window_layer(heads=6, kv_heads=3, dim=40, size=37, ff=80, scale=0.21),
              R.window_layer(heads=3, kv_heads=3, dim=8, size=64, ff=None),
              R.latent_layer(heads=4, dim=16, rot_dim=32, vdim=16, q_rank=48, kv_rank=24, base=100.0, scale=0.3, ff=None)]
    return R.make_config(layers, width=72, vocab=97, streams=3, eps=1e-6, loop={"start": 1, "stop": 3, "times": 3})


def cfg_odd():
    """Sizes the vectorised and tensor-core kernels do not take: odd head sizes, an odd width, five streams, 40 query
    heads on one key/value head, a head of 130."""
    layers = [R.window_layer(heads=40, kv_heads=1, dim=6, size=33, ff=30), R.window_layer(heads=2, kv_heads=1, dim=130, size=5, ff=None),
              R.latent_layer(heads=7, dim=5, rot_dim=6, vdim=9, q_rank=11, kv_rank=13, ff=27),
              R.retention_layer(heads=1, dim=34, vdim=7, rot_dims=2), R.retention_layer(heads=3, dim=70, vdim=33, rot_dims=64)]
    return R.make_config(layers, width=51, vocab=61, streams=5, loop={"start": 3, "stop": 4, "times": 1})


CONFIGS = {"window": cfg_window, "latent": cfg_latent, "retention": cfg_retention, "loop": cfg_loop, "full": cfg_full, "odd": cfg_odd}


def _case(name, seed=0):
    config = CONFIGS[name]()
    return config, R.random_weights(config, seed)


# ------------------------------------------------------------------------------------------------------------ CPU tests
def test_oracle_attention_loop_equals_matrix_form():
    config, W = _case("full")
    toks = _tokens(41, config["vocab"], 1)
    try:
        R.FORM = "loop"
        a = R.forward(config, W, toks)
    finally:
        R.FORM = "matrix"
    assert (a - R.forward(config, W, toks)).abs().max() < 1e-9


def test_oracle_prefix_property():
    config, W = _case("full")
    toks = _tokens(50, config["vocab"], 2)
    full = R.forward(config, W, toks)
    assert (R.forward(config, W, toks[:17]) - full[:17]).abs().max() < 1e-9


def test_oracle_small_functions():
    assert [j for j in range(12) if R.sees_window(9, j, 4)] == [6, 7, 8, 9]
    x = torch.arange(1.0, 11.0, dtype=torch.float64)
    y = R.turn_halves(x, 5, 6, 100.0)
    assert torch.equal(y[6:], x[6:])
    assert abs(float(y[0]) - (1 * math.cos(5.0) - 4 * math.sin(5.0))) < 1e-12       # entry 0 turns with entry 3
    a = 5 * 100 ** (-2 / 6)
    assert abs(float(y[4]) - (5 * math.cos(a) + 2 * math.sin(a))) < 1e-12           # entry 1 turns with entry 4
    z = torch.randn(9, 2, 10, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    want = torch.stack([torch.stack([R.turn_halves(z[t, h], t, 6, 100.0) for h in range(2)]) for t in range(9)])
    assert (R.turn_all(z, 6, 100.0) - want).abs().max() < 1e-12
    q = torch.ones(2, 1, 1, dtype=torch.float64)
    v = torch.tensor([[[2.0]], [[4.0]]], dtype=torch.float64)
    o = R.sigmoid_attention(q, q * 0, v, 1, 1.0, [0.0], 5)
    assert o.flatten().tolist() == [1.0, 3.0]                                        # half of every visible value, no division
    o = R.retain(q, q, v, [0.5])
    assert o.flatten().tolist() == [2.0, 5.0]
    X = torch.tensor([[[1.0]], [[10.0]]], dtype=torch.float64)
    W = {"in": torch.tensor([1.0, 2.0]), "out": torch.tensor([3.0, 5.0]), "mix": torch.tensor([[1.0, 7.0], [0.5, 0.0]])}
    Y = R.sublayer(X, {n: t.double() for n, t in W.items()}, "", lambda u: 2 * u)
    assert Y.flatten().tolist() == [1.0 + 5.0 + 3 * 42.0, 7.0 + 5 * 42.0]            # mix is [from][to]
    assert R.layer_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3]


def test_registry_names_the_design():
    from llm_decoder.hybrid import DESIGNS, FEED_FORWARDS
    from llm_decoder.registry import MODEL_REGISTRY
    assert "Namudra" in MODEL_REGISTRY and DESIGNS["Namudra"]["wiring"] == "streams"
    assert set(DESIGNS["Namudra"]["mixers"]) == {"attention", "latent_attention", "retention"}
    assert set(DESIGNS["Namudra"]["ff"]) <= set(FEED_FORWARDS)


# ------------------------------------------------------------------------------------------------------------ GPU tests
@pytest.mark.gpu
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_each_mechanism(name, dtype):
    import llm_decoder as ld
    config, W = _case(name)
    toks = _tokens(85, config["vocab"], 3)
    eng = ld.Engine(_model(config, W, dtype))
    _close(_feed(eng, "a", toks, []), _oracle(name, config, W, toks), dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("name,runs", [("full", 9), ("loop", 6)])
def test_residual_after_every_layer_run(name, runs):
    """The sum of the streams after every layer run, and the logits of the steps with the hook installed."""
    import llm_decoder as ld
    config, W = _case(name)
    toks = _tokens(45, config["vocab"], 6)
    model = _model(config, W)
    seen = []
    model.layer_hook = lambda x: seen.append(x.double().cpu())
    got = ld.Engine(model).step([("a", toks, list(range(45)))])
    want = []
    logits = R.forward(config, W, toks, want)
    assert len(seen) == len(want) == runs
    for i, x in enumerate(seen):
        assert (x - want[i]).abs().max() < 3e-5 * max(1.0, want[i].abs().max().item()), f"layer run {i}"
    _close(got, logits)


CHANGES = {     # tensor or constant -> what becomes of it
    "pb": lambda c, W: W.update({"l2.mix.pb": (W["l2.mix.pb"].float() + 1.0).to(torch.bfloat16)}),
    "k.norm": lambda c, W: W.update({"l2.mix.k.norm": W["l2.mix.k.norm"].flip(0).contiguous()}),
    "q.norm": lambda c, W: W.update({"l2.mix.q.norm": (W["l2.mix.q.norm"].float() * 1.5).to(torch.bfloat16)}),
    "gate": lambda c, W: W.update({"l2.mix.g": W["l2.mix.g"].flip(0).contiguous()}),
    "mix transposed": lambda c, W: W.update({"l2.hc1.mix": W["l2.hc1.mix"].t().contiguous()}),
    "in": lambda c, W: W.update({"l1.hc2.in": W["l1.hc2.in"].flip(0).contiguous()}),
    "out": lambda c, W: W.update({"l3.hc1.out": W["l3.hc1.out"].flip(0).contiguous()}),
    "final": lambda c, W: W.update({"final.norm": (W["final.norm"].float() + 0.5).to(torch.bfloat16)}),
    "dkv.norm": lambda c, W: W.update({"l1.mix.dkv.norm": W["l1.mix.dkv.norm"].flip(0).contiguous()}),
    "window": lambda c, W: c["layers"][2]["mixer"]["mask"].update(size=36),
    "decay": lambda c, W: c["layers"][0]["mixer"].update(decay=[0.9, 1.0, 0.5, 0.995]),
    "rot.dims": lambda c, W: c["layers"][0]["mixer"]["rot"].update(dims=12),
    "base": lambda c, W: c["layers"][1]["mixer"]["rot"].update(base=50.0),
    "times": lambda c, W: c["loop"].update(times=2),
    "start": lambda c, W: c["loop"].update(start=2),
    "eps": lambda c, W: c["norm"].update(eps=0.05),
}


@pytest.mark.gpu
@pytest.mark.parametrize("name", list(CHANGES))
def test_every_constant_shows_in_the_logits(name):
    """Changing one tensor or constant of the model moves the oracle's logits AND the engine follows: none of them is
    left out on the way."""
    import llm_decoder as ld
    config, W = _case("full", seed=3)
    toks = _tokens(60, config["vocab"], 16)
    base = _oracle("full3", config, W, toks)
    W2, config2 = dict(W), json.loads(json.dumps(config))
    CHANGES[name](config2, W2)
    want = R.forward(config2, W2, toks)
    assert (want - base).abs().max() > 0.01
    _close(_feed(ld.Engine(_model(config2, W2)), "a", toks, [33]), want)


@pytest.mark.gpu
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prefill_equals_token_by_token(name):
    import llm_decoder as ld
    config, W = _case(name)
    toks = _tokens(70, config["vocab"], 4)
    eng = ld.Engine(_model(config, W))
    _close(_feed(eng, "a", toks, range(1, 70)), _oracle(name, config, W, toks))      # every token a step of its own


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[2, 4, 6, 9, 40], [15, 16, 17, 31, 33, 48, 64, 66], [1, 80], [63], [4, 5, 6, 41, 42, 43, 78],
                                  [36, 37, 38, 74, 75]])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_many_sizes(cuts, dtype):
    """Cuts at, before and after page borders (16 tokens), key steps (32, 64), scan staging steps (16) and the window (37),
    down to two tokens."""
    import llm_decoder as ld
    config, W = _case("full")
    toks = _tokens(90, config["vocab"], 5)
    eng = ld.Engine(_model(config, W, dtype))
    _close(_feed(eng, "a", toks, cuts), _oracle("full", config, W, toks), dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["full", "loop"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_of_unequal_requests(name, dtype):
    """Four requests of unequal length advance together: portions next to single tokens, one sitting out a step; and each
    equals the same request alone."""
    import llm_decoder as ld
    config, W = _case(name)
    reqs = {r: _tokens(n, config["vocab"], 10 + i) for i, (r, n) in enumerate([("a", 70), ("b", 33), ("c", 5), ("d", 51)])}
    plan = [[("a", 40), ("b", 2)], [("a", 1), ("b", 17), ("c", 5)], [("a", 1), ("d", 30)], [("a", 1), ("b", 1), ("d", 1)],
            [("b", 13), ("d", 20), ("a", 27)]]
    eng = ld.Engine(_model(config, W, dtype))
    at = {r: 0 for r in reqs}
    got = {r: [] for r in reqs}
    for step in plan:
        entries = []
        for r, n in step:
            entries.append((r, reqs[r][at[r]:at[r] + n], list(range(n))))
            at[r] += n
        out = eng.step(entries)
        o = 0
        for r, n in step:
            got[r].append(out[o:o + n])
            o += n
    for r in reqs:
        assert at[r] == len(reqs[r])
        _close(torch.cat(got[r], 0), _oracle(name, config, W, reqs[r]), dtype)
        alone = _feed(ld.Engine(_model(config, W, dtype)), r, reqs[r], [])
        _close(torch.cat(got[r], 0), alone.double().cpu(), dtype, tol=1e-4, bf16_tol=0.04)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_large_decode_batch(dtype):
    """80 sequences of unequal length decode two tokens side by side: enough (token, key/value head) pairs for the
    tensor-core kernel of decoded tokens, windows of one key up to the whole sequence."""
    import llm_decoder as ld
    config = R.make_config([R.window_layer(heads=6, kv_heads=2, dim=16, size=21), R.latent_layer(heads=3, dim=8, rot_dim=8, kv_rank=16),
                            R.window_layer(heads=4, kv_heads=2, dim=40, size=70, ff=None), R.retention_layer(heads=2, dim=8, vdim=8, rot_dims=8)],
                           width=64, streams=2)
    W = R.random_weights(config, 11)
    lens = [1 + (i * 7) % 90 for i in range(80)]
    seqs = [_tokens(n + 2, config["vocab"], 500 + i) for i, n in enumerate(lens)]
    eng = ld.Engine(_model(config, W, dtype, max_tokens=80 * 96, max_seqs=80))
    eng.step([(i, q[:-2], []) for i, q in enumerate(seqs)])
    got = [eng.step([(i, q[t:t + 1] if t + 1 else q[t:], [0]) for i, q in enumerate(seqs)]) for t in (-2, -1)]
    want = [R.forward(config, W, q)[-2:] for q in seqs]
    for t in (0, 1):
        _close(got[t], torch.stack([w[t] for w in want]), dtype)


@pytest.mark.gpu
def test_wanted_rows_and_steps_without_any():
    """Logits of some rows, in any order and twice, and steps in which nothing is wanted (their cache and state stay)."""
    import llm_decoder as ld
    config, W = _case("full")
    a, b = _tokens(30, config["vocab"], 70), _tokens(21, config["vocab"], 71)
    eng = ld.Engine(_model(config, W))
    assert eng.step([("a", a[:12], []), ("b", b[:1], [])]).shape == (0, config["vocab"])
    out = eng.step([("b", b[1:], [19, 0, 0]), ("a", a[12:], [3])])
    wa, wb = _oracle("full", config, W, a), _oracle("full", config, W, b)
    _close(out, torch.stack([wb[20], wb[1], wb[1], wa[15]]))


@pytest.mark.gpu
def test_slots_and_pages_are_used_again():
    """A pool of 160 tokens and two slots serves six requests one after another and interleaved: freed pages and slots
    come back (dirty) and the next request must not see the keys or states they held."""
    import llm_decoder as ld
    config, W = _case("full")
    model = _model(config, W, max_tokens=160, max_seqs=2)
    assert len(model.states._kv) == 2 * 3 + 2               # the two looped layers have a pool per pass
    eng = ld.Engine(model)
    seqs = [_tokens(n, config["vocab"], 20 + i) for i, n in enumerate([90, 60, 33, 100, 17, 59])]
    out = eng.step([("r0", seqs[0][:50], list(range(50))), ("r1", seqs[1][:10], list(range(10)))])
    g0, g1 = [out[:50]], [out[50:]]
    out = eng.step([("r1", seqs[1][10:], list(range(50))), ("r0", seqs[0][50:], list(range(40)))])
    g1.append(out[:50])
    g0.append(out[50:])
    _close(torch.cat(g0), _oracle("full", config, W, seqs[0]))
    _close(torch.cat(g1), _oracle("full", config, W, seqs[1]))
    assert model.states.free_slots() == 0 and model.states.free_tokens() == 0
    with pytest.raises(RuntimeError):
        eng.step([("r2", [1], [0])])                 # no slot left
    eng.finish("r0")
    eng.finish("r1")
    assert model.states.free_slots() == 2 and model.states.free_tokens() == 160
    for i in (2, 3, 4, 5):
        _close(_feed(eng, f"r{i}", seqs[i], [len(seqs[i]) // 2]), _oracle("full", config, W, seqs[i]))
        eng.finish(f"r{i}")


@pytest.mark.gpu
def test_looped_retention_keeps_a_state_per_pass():
    """Slots used again under a looped retention layer: every pass starts from its own zero state."""
    import llm_decoder as ld
    config, W = _case("loop")
    eng = ld.Engine(_model(config, W, max_tokens=96, max_seqs=1))
    for i, n in enumerate((60, 3, 41)):
        toks = _tokens(n, config["vocab"], 80 + i)
        _close(_feed(eng, i, toks, [n // 3]), _oracle("loop", config, W, toks))
        eng.finish(i)


@pytest.mark.gpu
@pytest.mark.parametrize("tile_size", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_window_edges_and_far_keys_long_sequence(tile_size, dtype):
    """300 tokens through a window of 70, latent attention and retention with slow decay: prompts cut around page borders
    and the window, then 40 decoded tokens that slide the window over decoded tokens."""
    import llm_decoder as ld
    config = R.make_config([R.window_layer(heads=4, kv_heads=1, dim=32, size=70, scale=0.5), R.latent_layer(heads=4, dim=16, rot_dim=8, scale=0.5),
                            R.retention_layer(heads=2, dim=16, vdim=32, rot_dims=16, decay=[0.9999, 0.97])], width=64, vocab=80, streams=2)
    W = R.random_weights(config, 7)
    toks = _tokens(300, config["vocab"], 8)
    want = _oracle("edges", config, W, toks)
    eng = ld.Engine(_model(config, W, dtype, tile_size=tile_size))
    cuts = [5, 6, 69, 70, 71, 75, 77, 127, 129, 135, 192, 255, 256] + list(range(260, 300))
    _close(_feed(eng, "a", toks, cuts), want, dtype)
    eng.finish("a")
    _close(_feed(eng, "b", toks, [5, 290]), want, dtype)


def _needle_model(kind, size=0):
    """One layer of one head whose key map got a rank-one term: the needle token's key lands on the probe token's query, so
    the needle takes almost all the weight of the probe -- where the probe sees it.  'window': keys are normed, so the head's
    bias pushes every other weight towards zero.  'latent' and 'retention': the term reads a
    direction in which only the needle token has a component, and lives in the dimensions the rotation leaves alone;
    'retention': nothing normalises the sum over the others, and the decay is one."""
    p, needle, probe = "l0.mix.", 7, 11
    if kind == "window":
        config = R.make_config([R.window_layer(heads=1, kv_heads=1, dim=24, size=size, scale=0.8, ff=None)], width=32, vocab=40)
    elif kind == "latent":
        config = R.make_config([R.latent_layer(heads=1, dim=20, rot_dim=4, kv_rank=48, scale=1.0, ff=None)], width=64, vocab=40)
    else:
        config = R.make_config([R.retention_layer(heads=1, dim=20, vdim=16, rot_dims=4, decay=[1.0])], width=64, vocab=40)
    W = R.random_weights(config, 9)
    D = {k: v.double() for k, v in W.items()}
    eps = config["norm"]["eps"]
    h = R.norm1p(D["embed"][[needle, probe]] * D["l0.hc1.in"].sum(), D["l0.norm1"], eps)
    if kind == "latent":
        c = config["layers"][0]["mixer"]
        q = ((R.rms(h[1] @ D[p + "dq"].T, eps) * D[p + "dq.norm"]) @ D[p + "uq"].T)[:c["dim"]]
        every = R.norm1p(D["embed"] * D["l0.hc1.in"].sum(), D["l0.norm1"], eps)
        lat = R.rms(every @ D[p + "dkv"].T[:, :c["kv_rank"]], eps) * D[p + "dkv.norm"]
        W[p + "uk"] = (D[p + "uk"] * 0.1 + 18.0 * torch.outer(q / (q @ q), torch.linalg.pinv(lat)[:, needle])).to(torch.bfloat16)
        return config, W, needle, probe
    q = D[p + "q"] @ h[1]
    gain, direction = 16.0, h[0] / (h[0] @ h[0])
    if kind == "window":
        W[p + "q.norm"] = W[p + "k.norm"] = torch.ones(24, dtype=torch.bfloat16)
        W[p + "pb"] = torch.full((1,), -9.0, dtype=torch.bfloat16)
    else:
        q[:4] = 0.0
        gain = 1000.0
        direction = torch.linalg.pinv(R.norm1p(D["embed"] * D["l0.hc1.in"].sum(), D["l0.norm1"], eps))[:, needle]
    W[p + "k"] = (D[p + "k"] * 0.2 + gain * torch.outer(q / (q @ q), direction)).to(torch.bfloat16)
    return config, W, needle, probe


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [48, 17, 1, 64, 33])
def test_single_key_at_the_window_edge(size, dtype):
    """The needle sits at the last position the probe still sees or at the first it does not; the probe comes at the end of
    a prompt portion, or decoded alone.  The test first proves that the placements give different logits."""
    import llm_decoder as ld
    config, W, needle, probe = _needle_model("window", size)
    others = [t for t in range(40) if t not in (needle, probe)]
    rnd = random.Random(3)
    n = 3 * size + 5                                        # the probe's position
    results = {}
    for where in (max(n - size + 1, 0) if size > 1 else n - 1, n - size):
        toks = [rnd.choice(others) for _ in range(n)] + [probe]
        toks[where] = needle
        want = R.forward(config, W, toks)
        results[where] = want[-1]
        for cuts in ([n], [], [where, where + 1, n - 1, n]):
            eng = ld.Engine(_model(config, W, dtype))
            _close(_feed(eng, "a", toks, cuts), want, dtype)
    if size > 1:
        assert (results[n - size + 1] - results[n - size]).abs().max() > 0.3


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["latent", "retention"])
@pytest.mark.parametrize("where", [0, 15, 16, 31, 32, 140])
def test_single_far_key_among_hundreds(kind, where):
    """400 tokens: one key, far back, takes the probe's weight; without it the logits differ."""
    import llm_decoder as ld
    config, W, needle, probe = _needle_model(kind)
    others = [t for t in range(40) if t not in (needle, probe)]
    rnd = random.Random(where)
    toks = [rnd.choice(others) for _ in range(400)] + [probe]
    without = R.forward(config, W, toks)[-1]
    toks[where] = needle
    want = R.forward(config, W, toks)
    assert (want[-1] - without).abs().max() > 0.3
    for cuts in ([400], [390], [where + 1, 399, 400]):
        _close(_feed(ld.Engine(_model(config, W)), "a", toks, cuts), want)


@pytest.mark.gpu
def test_first_tokens():
    import llm_decoder as ld
    for name in ("full", "odd"):
        config, W = _case(name)
        for n in (1, 2, 3):
            toks = _tokens(n, config["vocab"], 30 + n)
            eng = ld.Engine(_model(config, W))
            _close(_feed(eng, "a", toks, []), _oracle(name, config, W, toks))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portion_and_long_decoding(dtype):
    """A 560-token portion (chunked scan) followed by 150 decoded tokens; the same request again cut at 300."""
    import llm_decoder as ld
    config, W = _case("full")
    toks = _tokens(710, config["vocab"], 40)
    want = _oracle("full", config, W, toks)
    eng = ld.Engine(_model(config, W, dtype))
    _close(_feed(eng, "a", toks, [560] + list(range(561, 710))), want, dtype, tol=1.5e-3)
    eng.finish("a")
    _close(_feed(eng, "b", toks, [300, 301, 700]), want, dtype, tol=1.5e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portion_beside_short_ones_in_one_step(dtype):
    """A 300-token portion (chunked scan for the whole batch) beside a decoded token, a two-token portion and a first one."""
    import llm_decoder as ld
    config, W = _case("full")
    seqs = {"a": _tokens(340, config["vocab"], 90), "b": _tokens(52, config["vocab"], 91), "c": _tokens(20, config["vocab"], 92),
            "d": _tokens(7, config["vocab"], 93)}
    eng = ld.Engine(_model(config, W, dtype))
    start = {"a": 40, "b": 50, "c": 18}
    eng.step([(r, seqs[r][:n], []) for r, n in start.items()])
    nxt = [("b", 1), ("a", 300), ("d", 7), ("c", 2)]
    out = eng.step([(r, seqs[r][start.get(r, 0):start.get(r, 0) + n], list(range(n))) for r, n in nxt])
    o = 0
    for r, n in nxt:
        lo = start.get(r, 0)
        _close(out[o:o + n], R.forward(config, W, seqs[r][:lo + n])[lo:], dtype)
        o += n


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype):
    """Scheduler: five prompts of unequal length on four slots with a small token budget (chunked prompts, continuous
    batching, slot reuse); greedy tokens equal the oracle's argmax at every step (float32), and the teacher-forced
    logits stay close (bfloat16)."""
    import llm_decoder as ld
    config, W = _case("full")
    prompts = [_tokens(n, config["vocab"], 50 + i) for i, n in enumerate([37, 5, 64, 18, 2])]
    model = _model(config, W, dtype, max_tokens=512, max_seqs=4)
    outs = ld.generate(model, prompts, 12, max_batch_tokens=48)
    for p, o in zip(prompts, outs):
        assert o[:len(p)] == p and len(o) == len(p) + 12
        logits = R.forward(config, W, o[:-1])
        for t in range(len(p) - 1, len(o) - 1):
            if dtype == "float32":
                top2 = logits[t].topk(2).values
                if float(top2[0] - top2[1]) > 1e-3:                 # no test on a near tie
                    assert int(logits[t].argmax()) == o[t + 1]
            else:
                assert float(logits[t].max() - logits[t, o[t + 1]]) < 0.3


def _random_config(rnd):
    """Layer count and order, the loop, every size and constant drawn at random."""
    layers = []
    for _ in range(rnd.randint(2, 6)):
        ff = rnd.choice([None, None, 8, 30, 64, 100])
        kind = rnd.randrange(3)
        if kind == 0:
            kv = rnd.choice([1, 2, 3])
            layers.append(R.window_layer(heads=kv * rnd.randint(1, 4), kv_heads=kv, dim=rnd.choice([8, 12, 16, 24, 33, 64]),
                                         size=rnd.randint(1, 90), scale=rnd.uniform(0.1, 0.5), ff=ff))
        elif kind == 1:
            layers.append(R.latent_layer(heads=rnd.randint(1, 9), dim=rnd.choice([8, 12, 16, 24, 20]), rot_dim=rnd.choice([2, 4, 8, 16, 40]),
                                         vdim=rnd.choice([8, 16, 40, 20, 6]), q_rank=rnd.choice([8, 24, 33]),
                                         kv_rank=rnd.choice([8, 16, 20, 64, 72]), base=rnd.choice([50.0, 10000.0, 500000.0]),
                                         scale=rnd.uniform(0.1, 0.4), ff=ff))
        else:
            H, dim = rnd.randint(1, 5), rnd.choice([8, 12, 16, 24, 66])
            layers.append(R.retention_layer(heads=H, dim=dim, vdim=rnd.choice([8, 16, 40, 20, 6]), rot_dims=rnd.randrange(2, dim + 1, 2),
                                            base=rnd.choice([50.0, 10000.0, 500000.0]),
                                            decay=[rnd.choice([1.0, 0.999, 0.98, 0.8]) for _ in range(H)], ff=ff))
    a = rnd.randrange(len(layers))
    loop = rnd.choice([None, {"start": a, "stop": rnd.randint(a + 1, len(layers)), "times": rnd.randint(1, 4)}])
    return R.make_config(layers, width=rnd.choice([40, 64, 72, 96, 50, 51]), vocab=rnd.choice([61, 97, 128]), streams=rnd.randint(1, 6),
                         eps=rnd.choice([1e-5, 1e-6, 1e-3]), loop=loop)


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(12))
def test_random_configurations_in_random_schedules(seed):
    """Three requests of a randomly drawn model advance in random portions (1 to 100 tokens, some sitting out) through
    one engine; float32 and bfloat16 against the oracle at every position."""
    import llm_decoder as ld
    rnd = random.Random(seed)
    config = _random_config(rnd)
    W = R.random_weights(config, seed)
    reqs = {r: _tokens(n, config["vocab"], 100 * seed + i)
            for i, (r, n) in enumerate((("a", rnd.randint(120, 300)), ("b", rnd.randint(2, 90)), ("c", rnd.randint(1, 40))))}
    plan, at = [], {r: 0 for r in reqs}
    while any(at[r] < len(reqs[r]) for r in reqs):
        step = []
        for r in reqs:
            left = len(reqs[r]) - at[r]
            if left and rnd.random() < 0.8:
                n = min(left, rnd.choice([1, 1, 2, 3, 17, 64, 100]))
                step.append((r, at[r], n))
                at[r] += n
        if step:
            plan.append(step)
    want = {r: R.forward(config, W, reqs[r]) for r in reqs}
    for dtype in ("float32", "bfloat16"):
        eng = ld.Engine(_model(config, W, dtype, max_tokens=640, max_seqs=3))
        got = {r: [] for r in reqs}
        for step in plan:
            out = eng.step([(r, reqs[r][lo:lo + n], list(range(n))) for r, lo, n in step])
            o = 0
            for r, _lo, n in step:
                got[r].append(out[o:o + n])
                o += n
        for r in reqs:
            _close(torch.cat(got[r], 0), want[r], dtype, tol=1e-3, bf16_tol=0.12)


# ---- kernels alone -----------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv_heads,dim", [(4, 2, 16), (6, 1, 96), (8, 2, 64), (3, 3, 40), (2, 1, 128), (9, 1, 24), (2, 2, 7)])
@pytest.mark.parametrize("weights,shared,gate,bias,size", [("sigmoid", True, True, True, 37), ("sigmoid", False, False, False, 200),
                                                           ("softmax", True, True, False, 5), ("softmax", False, True, True, 64),
                                                           ("sigmoid", True, False, True, 1)])
def test_attention_kernels_alone(heads, kv_heads, dim, weights, shared, gate, bias, size):
    """The float tile kernel, the streaming single-token kernel and the tensor-core kernel over the same paged pool (pages
    handed out in a scattered order) against attention written out in float64: pa_qk_norm_kv_append fills the pool (keys
    normed beside values of their own, or one row per key with its inverse root mean square), then sigmoid or softmax
    weights in a window, with a number per head on the score and the gate on the output.  A 150-token portion that starts at
    position 70 of its sequence, a first token, a two-token portion at positions 63 and 64, a single token at position 219."""
    from llm_decoder import _cabi
    from llm_decoder.seq_state import SequenceStateCache
    lib, dev, s = _cabi.lib(), torch.device("cuda"), _cabi.stream()
    g = torch.Generator().manual_seed(heads * 7 + dim)
    per, scale, eps = heads // kv_heads, 0.3, 1e-5
    ctx, new = [70, 0, 63, 219], [150, 1, 2, 1]             # tokens already cached / of this step
    gq, gk, hb = torch.rand(dim, generator=g) + 0.5, torch.rand(dim, generator=g) + 0.5, torch.randn(heads, generator=g)
    qc, kc = heads * dim, kv_heads * dim
    cols = qc + kc * (1 if shared else 2) + qc
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        states = SequenceStateCache(4, 1024, 16, dev)
        kv = states.add_kv_layer(kv_heads, dim, 0 if shared else dim, "f32" if dtype == torch.float32 else "bf16", key_scale=shared)
        slots = [states.alloc() for _ in range(4)]
        for rnd_ in range(14):                              # interleave the sequences' growth so that their pages interleave
            for i in [2, 0, 3, 1]:
                n = min(16, ctx[i] - rnd_ * 16)
                if n > 0:
                    states.extend(slots[i], n)
        X = [torch.randn(ctx[i] + new[i], cols, generator=g).to(dtype) for i in range(4)]
        pt = kv.page_table_
        table = pt.device_data()
        gain_q, gain_k = (gq * gk if shared else gq).to(dev), gk.to(dev)

        def append(rows, slot, pos):
            assert lib.pa_qk_norm_kv_append(rows.data_ptr(), rows.stride(0), 0, qc, qc + kc, heads, kv_heads, dim, dim, gain_q.data_ptr(),
                                            gain_k.data_ptr(), eps, kv.key_buffer_.data_ptr(),
                                            None if shared else kv.value_buffer_.data_ptr(), _cabi.ptr(kv.key_scale_), table.data_ptr(),
                                            pt.num_beams_, pt.num_tiles_, kv.total_pages_, kv.tile_size_, slot.data_ptr(), pos.data_ptr(),
                                            rows.shape[0], rows.element_size(), s) == 0
        for i in range(4):
            if ctx[i]:
                append(X[i][:ctx[i]].to(dev), torch.full((ctx[i],), slots[i], dtype=torch.int32, device=dev),
                       torch.arange(ctx[i], dtype=torch.int32, device=dev))
        table = pt.device_data()
        batch = states.make_batch([(slots[i], [0] * new[i]) for i in range(4)])
        table = pt.device_data()
        proj = torch.cat([X[i][ctx[i]:] for i in range(4)], 0).to(dev)
        append(proj, batch.row_slot, batch.row_pos)
        want = []
        for i in range(4):
            x = X[i].double()
            T = ctx[i] + new[i]
            q = R.rms(x[ctx[i]:, :qc].reshape(new[i], heads, dim), eps) * gq.double()
            kraw = x[:, qc:qc + kc].reshape(T, kv_heads, dim)
            k = R.rms(kraw, eps) * gk.double()
            v = kraw if shared else x[:, qc + kc:qc + 2 * kc].reshape(T, kv_heads, dim)
            d = torch.arange(ctx[i], T)[:, None] - torch.arange(T)[None, :]
            vis = (d >= 0) & (d < size)
            out = torch.zeros(new[i], heads, dim, dtype=torch.float64)
            for h in range(heads):
                sc = q[:, h] @ k[:, h // per].T * scale + (float(hb[h]) if bias else 0.0)
                w = R.sigmoid(sc) * vis if weights == "sigmoid" else torch.softmax(sc.masked_fill(~vis, -math.inf), -1)
                out[:, h] = w @ v[:, h // per]
            out = out.reshape(new[i], qc)
            want.append(out * R.sigmoid(x[ctx[i]:, cols - qc:]) if gate else out)
        want = torch.cat(want, 0)
        tt = lib.pa_masked_attention_tile_tokens(heads, kv_heads)
        mt = lib.pa_masked_attention_mma_tile_tokens(dim, dim, proj.element_size())
        hbd = hb.to(dev)
        vals = kv.key_buffer_ if shared else kv.value_buffer_
        # single tokens: the tile kernel, the streaming kernel, and (where the shape is served) heads as rows on the tensor cores
        for use_mma, single in ((0, 0), (mt, 1)) + (((mt, 3),) if mt else ()):
            out = torch.zeros(sum(new), qc, dtype=dtype, device=dev)
            for kind, group in batch.query_tiles(tt, use_mma, 16).items():
                if group is None:
                    continue
                tiles, ntiles, _longest = group
                args = lambda kd: (proj.data_ptr(), proj.stride(0), 0, kv.key_buffer_.data_ptr(), vals.data_ptr(), table.data_ptr(),  # noqa: E731
                                   pt.num_beams_, pt.num_heads_, pt.num_tiles_, kv.total_pages_, kv.tile_size_, tiles.data_ptr(), ntiles,
                                   heads, dim, dim, scale, 0.0, 1, size, 0, 0, None, 0, None, None, None, _cabi.ptr(kv.key_scale_),
                                   1 if weights == "sigmoid" else 0, hbd.data_ptr() if bias else None, proj.data_ptr() if gate else None,
                                   proj.stride(0), cols - qc, out.data_ptr(), proj.element_size(), kd, s)
                rc = lib.pa_masked_attention_gated(*args(single if kind == 1 else kind))
                assert rc == 0, (kind, rc)
            err = (out.double().cpu() - want).abs().max().item()
            assert err < tol * max(1.0, want.abs().max().item()), (dtype, use_mma, err)


@pytest.mark.gpu
@pytest.mark.parametrize("heads,dim,vdim,rot_dims", [(2, 16, 8, 16), (4, 24, 40, 10), (1, 150, 70, 2), (3, 64, 64, 64), (2, 5, 3, 4),
                                                     (1, 300, 20, 300), (2, 8, 8, 0)])
def test_rotated_scan_kernel_alone(heads, dim, vdim, rot_dims):
    """Portions of 1, 3, 40 and 300 tokens at positions 0, 5, 63 and 1000 from random states in slots 2, 0, 3, 1: the walk in
    order and the chunked three-pass form, queries and keys turned and keys scaled inside, against the recurrence in float64;
    then the norm per head with the silu gate."""
    from llm_decoder import _cabi
    from llm_decoder.seq_state import SequenceStateCache
    lib, dev, s = _cabi.lib(), torch.device("cuda"), _cabi.stream()
    g = torch.Generator().manual_seed(heads * 100 + dim)
    lens, slots, first, base = [1, 3, 40, 300], [2, 0, 3, 1], [0, 5, 63, 1000], 500.0
    decay = torch.rand(heads, generator=g) * 0.2 + 0.8
    k_scale, eps, cols = dim ** -0.5, 1e-5, heads * (2 * dim + 2 * vdim)
    pos = torch.cat([torch.arange(p, p + n) for p, n in zip(first, lens)])
    for dtype in (torch.float32, torch.bfloat16):
        x = torch.randn(sum(lens), cols, generator=g).to(dtype)
        state0 = torch.randn(4, heads, dim, vdim, generator=g)
        xd = x.double()
        q, k, v = (xd[:, a:b].reshape(-1, heads, n) for a, b, n in ((0, heads * dim, dim), (heads * dim, 2 * heads * dim, dim),
                                                                    (2 * heads * dim, 2 * heads * dim + heads * vdim, vdim)))
        half = rot_dims // 2
        ang = pos.double()[:, None] * torch.tensor([base ** (-2.0 * i / rot_dims) for i in range(half)], dtype=torch.float64)
        co, si = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        turn = lambda z: torch.cat([z[..., :half] * co - z[..., half:rot_dims] * si, z[..., half:rot_dims] * co + z[..., :half] * si,  # noqa: E731
                                    z[..., rot_dims:]], -1)
        q, k = turn(q), turn(k) * k_scale
        want, state = torch.zeros(sum(lens), heads, vdim, dtype=torch.float64), state0.double().clone()
        r = 0
        for i, n in enumerate(lens):
            for t in range(r, r + n):
                state[i] = decay.double()[:, None, None] * state[i] + k[t][:, :, None] * v[t][:, None, :]
                want[t] = (state[i] * q[t][:, :, None]).sum(1)
            r += n
        rope = None
        if rot_dims:
            rope = torch.empty(sum(lens), half, 2, device=dev)
            rp = pos.to(torch.int32).to(dev)
            assert lib.pa_rope_table(rp.data_ptr(), sum(lens), rot_dims, base, rope.data_ptr(), s) == 0
        X, dec = x.to(dev), decay.to(dev)
        for chunk in (0, 64):
            states = SequenceStateCache(4, 1024, 16, dev)
            st = states.add_state(heads * dim * vdim)
            for _ in slots:
                states.alloc()
            batch = states.make_batch([(sl, [0] * n) for sl, n in zip(slots, lens)])
            for i, sl in enumerate(slots):
                st[sl] = state0[i].reshape(-1).to(dev)
            items, n, s0, sn = batch.chunk_items(chunk)
            ws = torch.empty(lib.pa_decay_scan_workspace_bytes(n, heads, dim, vdim) if chunk else 1, dtype=torch.uint8, device=dev)
            out = torch.empty(sum(lens), heads * vdim, device=dev)
            assert lib.pa_decay_scan_rotated(X.data_ptr(), cols, 0, X.data_ptr(), cols, heads * dim, X.data_ptr(), cols, 2 * heads * dim,
                                             heads, heads, dim, vdim, 0, dec.data_ptr(), None, 0, 0, None, None, None, _cabi.ptr(rope),
                                             rot_dims, k_scale, st.data_ptr(), out.data_ptr(), heads * vdim, items.data_ptr(), n,
                                             s0.data_ptr(), sn.data_ptr(), batch.seq_slot.data_ptr(), batch.num_seqs, 1 if chunk else 0,
                                             ws.data_ptr(), ws.numel(), X.element_size(), s) == 0
            assert (out.double().cpu().reshape(want.shape) - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item())
            for i, sl in enumerate(slots):
                assert (st[sl].double().cpu().reshape(heads, dim, vdim) - state[i]).abs().max() < 2e-5 * max(1.0, state.abs().max().item())
        gated = torch.empty(sum(lens), heads * vdim, dtype=dtype, device=dev)
        assert lib.pa_gated_rms_norm(out.data_ptr(), sum(lens), heads * vdim, heads, X.data_ptr(), cols, cols - heads * vdim, 3, None, eps,
                                     gated.data_ptr(), X.element_size(), s) == 0
        ref = R.rms(want, eps).reshape(sum(lens), -1) * R.silu(xd[:, cols - heads * vdim:])
        assert (gated.double().cpu() - ref).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2) * ref.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8, 11, 16])
@pytest.mark.parametrize("width", [64, 51, 1300])
def test_residual_streams_kernel_alone(streams, width):
    """Update from one shared row and from streams of their own, in place and aside, with and without an output to add; the
    weighted sum, its norm, and the same for chosen rows only."""
    from llm_decoder import _cabi
    lib, dev, s = _cabi.lib(), torch.device("cuda"), _cabi.stream()
    g = torch.Generator().manual_seed(streams * 1000 + width)
    rows, S, eps = 7, streams, 1e-4
    a, b, M = torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(S, S, generator=g)
    gain = torch.rand(width, generator=g) + 0.5
    ad, bd, Md, gd = a.to(dev), b.to(dev), M.to(dev), gain.to(dev)
    pick = torch.tensor([6, 0, 6, 3], dtype=torch.int32)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        e = 4 if dtype == torch.float32 else 2
        y = torch.randn(rows, width, generator=g).to(dtype)
        yd = y.to(dev)
        for n in {1, S}:
            x = torch.randn(rows, n, width, generator=g)
            old = x.double().expand(rows, S, width)
            new = torch.einsum("st,rsw->rtw", M.double(), old) + b.double()[None, :, None] * y.double()[:, None]
            for given in (True, False):
                cur = new if given else old
                xd = x.to(dev)
                dst = None if not given else xd if n == S else torch.empty(rows, S, width, device=dev)
                u, h = torch.empty(rows, width, device=dev), torch.empty(rows, width, dtype=dtype, device=dev)
                yp, mp, bp = (yd.data_ptr(), Md.data_ptr(), bd.data_ptr()) if given else (None, None, None)
                final = torch.empty(4, width, dtype=dtype, device=dev)
                assert lib.pa_streams_add_norm(xd.data_ptr(), n, None, 4, S, width, yp, mp, bp, None, eps, gd.data_ptr(), None,
                                               final.data_ptr(), pick.to(dev).data_ptr(), e, s) == 0
                assert lib.pa_streams_add_norm(xd.data_ptr(), n, _cabi.ptr(dst), rows, S, width, yp, mp, bp, ad.data_ptr(), eps,
                                               gd.data_ptr(), u.data_ptr(), h.data_ptr(), None, e, s) == 0
                total = cur.sum(1)[pick.long()]
                assert (final.double().cpu() - R.rms(total, eps) * gain.double()).abs().max() < tol * 5
                want = torch.einsum("t,rtw->rw", a.double(), cur)
                assert (u.double().cpu() - want).abs().max() < 1e-5 * max(1.0, want.abs().max().item())
                assert (h.double().cpu() - R.rms(want, eps) * gain.double()).abs().max() < tol * 5
                if given:
                    assert (dst.double().cpu() - new).abs().max() < 1e-5 * max(1.0, new.abs().max().item())
    x = torch.zeros(1, 17, 4, device=dev)       # more streams than the kernel holds: refused, not cut off
    assert lib.pa_streams_add_norm(x.data_ptr(), 17, None, 1, 17, 4, None, None, None, None, eps, None, x.data_ptr(), None, None, 4,
                                   s) == _cabi.PA_ERR_UNSUPPORTED


@pytest.mark.gpu
@pytest.mark.parametrize("pairing", [0, 1])
@pytest.mark.parametrize("kv_rank,rot_dim,dims,q_rank", [(40, 16, 16, 24), (13, 6, 4, 33), (72, 2, 2, 8)])
def test_latent_append_and_query_rotation_alone(pairing, kv_rank, rot_dim, dims, q_rank):
    """pa_latent_norm_append (the query latent's norm beside the pool rows) and pa_rope_rows_paired, pairs of neighbours
    and of halves, at positions around page borders."""
    from llm_decoder import _cabi
    from llm_decoder.seq_state import SequenceStateCache
    lib, dev, s = _cabi.lib(), torch.device("cuda"), _cabi.stream()
    g = torch.Generator().manual_seed(kv_rank)
    ctx, new, base, eps, heads = [14, 0, 1000], [5, 1, 20], 300.0, 1e-5, 3
    rows = sum(new)
    pos = [p for c, n in zip(ctx, new) for p in range(c, c + n)]

    def turn(v, p):         # oracle layout: halves; neighbours are the same pairs written in another order
        order = list(range(0, dims, 2)) + list(range(1, dims, 2)) if pairing == 0 else list(range(dims))
        out = v.clone()
        out[order] = R.turn_halves(v[order], p, dims, base)
        return out
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        e = 4 if dtype == torch.float32 else 2
        states = SequenceStateCache(3, 2048, 16, dev)
        kv = states.add_kv_layer(1, kv_rank + rot_dim, 0, "f32" if e == 4 else "bf16")
        slots = [states.alloc() for _ in range(3)]
        for sl, n in zip(slots, ctx):
            if n:
                states.extend(sl, n)
        batch = states.make_batch([(sl, [0] * n) for sl, n in zip(slots, new)])
        cols = q_rank + kv_rank + rot_dim + 3
        x = torch.randn(rows, cols, generator=g).to(dtype)
        gq, gk = torch.rand(q_rank, generator=g) + 0.5, torch.rand(kv_rank, generator=g) + 0.5
        rope = torch.empty(rows, dims // 2, 2, device=dev)
        assert lib.pa_rope_table(batch.row_pos.data_ptr(), rows, dims, base, rope.data_ptr(), s) == 0
        X, cq, gqd, gkd = x.to(dev), torch.empty(rows, q_rank, dtype=dtype, device=dev), gq.to(dev), gk.to(dev)
        pt = kv.page_table_
        table = pt.device_data()
        assert lib.pa_latent_norm_append(kv.key_buffer_.data_ptr(), table.data_ptr(), pt.num_beams_, pt.num_tiles_, kv.total_pages_,
                                         kv.tile_size_, kv_rank, rot_dim, dims, pairing, X.data_ptr(), cols, q_rank, gkd.data_ptr(), eps,
                                         rope.data_ptr(), 0, q_rank, gqd.data_ptr(), cq.data_ptr(), q_rank, batch.row_slot.data_ptr(),
                                         batch.row_pos.data_ptr(), rows, e, s) == 0
        xd = x.double()
        assert (cq.double().cpu() - R.rms(xd[:, :q_rank], eps) * gq.double()).abs().max() < tol * 2
        pool = kv.key_buffer_.double().cpu().reshape(-1, 16, kv_rank + rot_dim)
        tab = table.cpu().reshape(pt.num_beams_, pt.num_tiles_)
        slot_of = [sl for sl, n in zip(slots, new) for _ in range(n)]
        for r in range(rows):
            got = pool[int(tab[slot_of[r], pos[r] // 16]), pos[r] % 16]
            lat = R.rms(xd[r, q_rank:q_rank + kv_rank], eps) * gk.double()
            assert (got[:kv_rank] - lat).abs().max() < tol * 2
            assert (got[kv_rank:] - turn(xd[r, q_rank + kv_rank:q_rank + kv_rank + rot_dim], pos[r])).abs().max() < tol * 2
        hs = rot_dim + 5                        # a head: 5 columns that stay, then the rotated part
        q = torch.randn(rows, 2 + heads * hs, generator=g).to(dtype)
        Q = q.to(dev)
        assert lib.pa_rope_rows_paired(Q.data_ptr(), Q.stride(0), 2 + 5, hs, heads, dims, rope.data_ptr(), pairing, rows, e, s) == 0
        Qc = Q.double().cpu()
        for r in range(rows):
            want = q[r].double().clone()
            for h in range(heads):
                a = 2 + h * hs + 5
                want[a:a + rot_dim] = turn(want[a:a + rot_dim], pos[r])
            assert (Qc[r] - want).abs().max() < tol * 2


# ---- configuration -------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
def test_a_single_residual_without_streams():
    """A config without 'streams' keeps one residual: x += f(N(x)).  The oracle's form of it: one stream, all weights one."""
    import llm_decoder as ld
    config, W = _case("full")
    config["streams"] = 1
    W = {n: (torch.ones([1] * t.dim(), dtype=t.dtype) if ".hc" in n else t) for n, t in W.items()}
    toks = _tokens(50, config["vocab"], 12)
    want = R.forward(config, W, toks)
    _close(_feed(ld.Engine(_model(config, W)), "a", toks, [20, 21]), want)
    bare = {k: v for k, v in config.items() if k != "streams"}
    plain = {n: t for n, t in W.items() if ".hc" not in n}
    _close(_feed(ld.Engine(_model(bare, plain)), "a", toks, [20, 21]), want)


@pytest.mark.gpu
def test_configuration_errors():
    def broken(name, change):
        config, W = _case(name)
        config = json.loads(json.dumps(config))
        change(config)
        with pytest.raises(ValueError):
            _model(config, W)
    broken("window", lambda c: c["layers"][0]["mixer"].update(vdim=8))           # values are the keys
    broken("window", lambda c: c["layers"][0]["mixer"].update(heads=6))          # the tensors have other rows
    broken("window", lambda c: c.update(streams=3))                              # the mixing weights are 2 x 2
    broken("retention", lambda c: c["layers"][0]["mixer"].update(decay=[0.5]))   # one decay per head
    broken("retention", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7))
    broken("latent", lambda c: c["layers"][0]["mixer"].update(kv_rank=8))
    broken("latent", lambda c: c["layers"][0].update(type="mamba2"))
    broken("loop", lambda c: c["loop"].update(stop=4))
    broken("full", lambda c: c["layers"][1]["mlp"].update(ff=8))


# ---- the command-line programs -------------------------------------------------------------------------------------------
@pytest.mark.gpu
def test_trace_runner_and_generate_programs(tmp_path):
    from llm_decoder.safetensors_io import save_file
    config, W = _case("full")
    mdir = tmp_path / "model"
    mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(config))
    save_file(W, str(mdir / "model.safetensors"))
    a, b = _tokens(40, config["vocab"], 60), _tokens(9, config["vocab"], 61)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [6]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[30:], "want": [9]}], "end": ["a"]}]
    out = tmp_path / "out"
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    import numpy as np
    wa, wb = R.forward(config, W, a), R.forward(config, W, b)
    for step, want in ((0, wa[[0, 29]]), (1, wb[[8]]), (2, wa[[39]])):
        _close(torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(want.shape[0], -1)), want)
    p = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", str(mdir), "--dtype", "float32", "--prompt",
                        ",".join(map(str, a[:12])), "--max-new-tokens", "5"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    toks = [int(t) for t in p.stdout.strip().splitlines()[-1].split(",")]
    assert toks[:12] == a[:12] and len(toks) == 17
    logits = R.forward(config, W, toks[:-1])
    for t in range(11, 16):
        top2 = logits[t].topk(2).values
        if float(top2[0] - top2[1]) > 1e-3:
            assert int(logits[t].argmax()) == toks[t + 1]
