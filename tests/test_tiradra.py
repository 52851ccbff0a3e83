"""The `Tiradra` design in the config-driven stack (llm_decoder.hybrid: token-pair embedding, two norms in parallel inside a
looped block whose passes add the embedding output and a step vector, attention on convolved, turned and then normed
projections, latent attention with a sink per head and an element gate, stretched rotations;
csrc/masked_attention.cu, latent_attention.cu, seq_ops.cu) against the plain float64 oracle (oracle/tiradra_ref.py), on
small random models of its own making.

The engine's logits at a position must equal the oracle's full recomputation whatever the cut into steps, the batch
around it, and the pages / slots in use."""
import json
import math
import os
import random
import subprocess

import pytest
import torch

from oracle import tiradra_ref as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 5e-4      # max abs error of float32 logits, per 4 units of their largest magnitude
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
        mid, worst = rel.median().item(), rel.max().item()
        assert math.isfinite(worst) and mid < bf16_tol and worst < 4 * bf16_tol, f"relative rms error {mid} (median), {worst} (worst)"


def _feed(engine, rid, tokens, cuts):
    """Feed `tokens` of one request in portions ending at `cuts`; returns logits of ALL positions."""
    outs, lo = [], 0
    for hi in list(cuts) + [len(tokens)]:
        if hi > lo:
            outs.append(engine.step([(rid, tokens[lo:hi], list(range(hi - lo)))]))
            lo = hi
    return torch.cat(outs, 0)


# ---- configurations: sizes and constants unlike each other -- one to nine key/value heads, head sizes that are no multiples of
# 8 or 32, one to eight taps, rotation over a part and over all of a head, with and without stretched frequencies, rot_dim
# above and below dim, vdim above and below dim, loops of one and several layers and none, one to three passes, layers
# without a feed-forward ------------------------------------------------------------------------------------------------
def cfg_attention():
    return R.make_config([R.attention_layer(heads=4, kv_heads=2, dim=24, vdim=16, taps=3, rot_dims=16)], width=64)


def cfg_latent():
    return R.make_config([R.latent_layer(heads=3, dim=8, rot_dim=16, vdim=20, kv_rank=40, base=500.0)], width=64)


def cfg_loop():
    return R.make_config([R.attention_layer(heads=2, kv_heads=1, dim=16, taps=2, ff=40), R.latent_layer(heads=2, dim=8, rot_dim=8, vdim=8, ff=None)],
                         width=48, loop={"start": 0, "stop": 2, "times": 3}, cap=None)


def cfg_full():
    layers = [R.latent_layer(heads=5, dim=24, rot_dim=8, vdim=40, kv_rank=72, ff=72, sc=R.scaling(3.0, 256, 20.0, 2.0)),
              R.attention_layer(heads=6, kv_heads=3, dim=40, vdim=24, taps=5, rot_dims=24, base=300.0, scale=0.31, ff=80),
              R.attention_layer(heads=3, kv_heads=3, dim=8, vdim=16, taps=2, sc=None, scale=0.6, ff=None),
              R.latent_layer(heads=4, dim=16, rot_dim=32, vdim=16, kv_rank=24, base=100.0, scale=0.3, ff=None),
              R.attention_layer(heads=8, kv_heads=2, dim=32, taps=4, rot_dims=32, sc=R.scaling(16.0, 32, 4.0, 0.25), scale=0.4, ff=56)]
    return R.make_config(layers, width=72, vocab=97, eps=1e-6, loop={"start": 1, "stop": 4, "times": 2}, buckets=53, mul_prev=17, mul_cur=101)


def cfg_odd():
    """Sizes the vectorised and tensor-core kernels do not take: odd head sizes, an odd width, one tap and eight, 40 query heads
    on one key/value head, a head of 130, a pair table of one row beside the first tokens' one."""
    layers = [R.attention_layer(heads=40, kv_heads=1, dim=6, vdim=5, taps=8, rot_dims=2, ff=30),
              R.attention_layer(heads=2, kv_heads=1, dim=130, vdim=67, taps=1, rot_dims=64, ff=None, scale=0.1),
              R.latent_layer(heads=7, dim=5, rot_dim=6, vdim=9, kv_rank=13, ff=27), R.attention_layer(heads=9, kv_heads=9, dim=7, vdim=9, taps=3, rot_dims=6)]
    return R.make_config(layers, width=51, vocab=61, loop={"start": 3, "stop": 4, "times": 1}, buckets=1, mul_prev=3, mul_cur=2)


CONFIGS = {"attention": cfg_attention, "latent": cfg_latent, "loop": cfg_loop, "full": cfg_full, "odd": cfg_odd}


def _case(name, seed=0):
    config = CONFIGS[name]()
    return config, R.random_weights(config, seed)


# ------------------------------------------------------------------------------------------------------------ CPU tests
def test_oracle_attention_loop_equals_matrix_form():
    config, W = _case("full")
    toks = _tokens(31, config["vocab"], 1)
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
    assert R.bigram_row(None, 4, 31, 5, 89) == 89 and R.bigram_row(3, 4, 31, 5, 89) == (93 + 20) % 89 and R.bigram_row(7, 0, 3, 9, 1) == 0
    W = {"embed": torch.tensor([[1.0], [2.0]]), "bigram": torch.tensor([[10.0], [20.0], [40.0], [80.0]])}
    e = R.embed(W, {"bigram": {"buckets": 3, "mul_prev": 2, "mul_cur": 1}}, [1, 0, 1])
    assert e.flatten().tolist() == [2.0 + 80.0, 1.0 + 40.0, 2.0 + 20.0]              # rows 3 (first), 2 * 1 + 0, 2 * 0 + 1
    x = torch.arange(1.0, 11.0, dtype=torch.float64)
    y = R.turn_neighbours(x, 5, {"dims": 6, "base": 100.0})
    assert torch.equal(y[6:], x[6:])
    assert abs(float(y[0]) - (1 * math.cos(5.0) - 2 * math.sin(5.0))) < 1e-12       # entry 0 turns with entry 1
    a = 5 * 100 ** (-2 / 6)
    assert abs(float(y[3]) - (4 * math.cos(a) + 3 * math.sin(a))) < 1e-12           # entry 2 turns with entry 3
    for rot in ({"dims": 6, "base": 100.0}, {"dims": 8, "base": 30.0, "scaling": R.scaling(4.0, 40, 4.0, 0.5)}):
        z = torch.randn(9, 2, 10, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
        want = torch.stack([torch.stack([R.turn_neighbours(z[t, h], t, rot) for h in range(2)]) for t in range(9)])
        assert (R.turn_all(z, rot) - want).abs().max() < 1e-12
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=torch.float64)
    assert R.short_convolution(u, torch.tensor([[2.0, 3.0]], dtype=torch.float64)).flatten().tolist() == [3.0, 32.0, 320.0]   # the LAST weight is the token's own
    q = torch.zeros(2, 1, 1, dtype=torch.float64)
    v = torch.tensor([[[6.0]], [[3.0]]], dtype=torch.float64)
    assert R.softmax_attention(q, q, v, 1.0).flatten().tolist() == [6.0, 4.5]
    assert torch.allclose(R.softmax_attention(q, q, v, 1.0, torch.zeros(1)).flatten(), torch.tensor([3.0, 3.0], dtype=torch.float64))
    assert R.layer_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [
        (0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]


def test_stretched_frequencies():
    """Fast pairs keep their frequency, slow ones are divided by the factor; worked out by hand for a small rotation, and the
    product's own function against the oracle's over many constants (borders of the ramp that fall outside the pairs, on each
    other, or on fractions)."""
    from llm_decoder.hybrid import rotation_scaling, scaled_frequencies
    f, mult = R.stretched_frequencies(8, 100.0, {"factor": 4.0, "original": 2 * math.pi * 10.0, "fast": 10.0, "slow": 0.1})
    # the pair that turns t times over the original positions: 8 ln(10 / t) / (2 ln 100), so 0 for fast and 4 for slow
    assert abs(mult - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    want = [100 ** (-i / 4) * ((i / 4) / 4.0 + 1 - i / 4) for i in range(4)]
    assert max(abs(a - b) for a, b in zip(f, want)) < 1e-12
    rnd = random.Random(0)
    for _ in range(200):
        dims, base = rnd.randrange(2, 130, 2), rnd.choice([20.0, 500.0, 10000.0, 1e6])
        sc = R.scaling(rnd.choice([1.0, 2.0, 40.0]), rnd.choice([4, 100, 4096, 65536]), rnd.choice([1.0, 32.0, 100.0]), rnd.choice([0.5, 1.0, 8.0]))
        a, ma = R.stretched_frequencies(dims, base, sc)
        b, mb = scaled_frequencies(dims, base, rotation_scaling({"scaling": sc}))
        assert abs(ma - mb) < 1e-12 and max(abs(x - y) / x for x, y in zip(a, b)) < 1e-12
    assert rotation_scaling({"dims": 8, "base": 10.0}) is None and rotation_scaling({"scaling": None}) is None


def test_batches_bring_the_previous_token():
    """A row's previous token: the one before it in the portion, the sequence's last one at a portion's start, -1 for a
    sequence's first token -- also when a slot is handed out again."""
    from llm_decoder.seq_state import SequenceStateCache
    st = SequenceStateCache(2, 256, 16, device="cpu")
    st.track_tokens = True
    a, b = st.alloc(), st.alloc()
    assert st.make_batch([(a, [5, 6, 7])]).prev_ids.tolist() == [-1, 5, 6]
    long = list(range(20, 40))
    assert st.make_batch([(b, long), (a, [9])]).prev_ids.tolist() == [-1] + long[:-1] + [7]
    assert st.make_batch([(a, [1, 2]), (b, [3])]).prev_ids.tolist() == [9, 1, 39]
    assert st.make_batch([(b, long)]).prev_ids.tolist() == [3] + long[:-1]
    st.free(a)
    assert st.make_batch([(st.alloc(), [8])]).prev_ids.tolist() == [-1]
    st.track_tokens = False
    assert st.make_batch([(b, [1])]).prev_ids is None


def test_portion_items():
    from llm_decoder.seq_state import SequenceStateCache
    st = SequenceStateCache(2, 256, 16, device="cpu")
    a, b = st.alloc(), st.alloc()
    st.make_batch([(a, [0] * 3)])
    items, n = st.make_batch([(b, [0] * 5), (a, [0] * 9)]).portion_items(4)
    assert n == 5 and items.tolist() == [[0, 4, b, 0, 5, 0], [4, 1, b, 4, 5, 4], [5, 4, a, 0, 9, 3], [9, 4, a, 4, 9, 7], [13, 1, a, 8, 9, 11]]


def test_registry_names_the_design():
    from llm_decoder.hybrid import DESIGNS, FEED_FORWARDS
    from llm_decoder.registry import MODEL_REGISTRY
    assert "Tiradra" in MODEL_REGISTRY and DESIGNS["Tiradra"]["wiring"] == "parallel_two_norms"
    assert set(DESIGNS["Tiradra"]["mixers"]) == {"attention", "latent_attention"}
    assert set(DESIGNS["Tiradra"]["ff"]) <= set(FEED_FORWARDS)


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
@pytest.mark.parametrize("name,runs", [("full", 8), ("loop", 6), ("odd", 4)])
def test_residual_after_every_layer_run(name, runs):
    """The residual after every layer run (before what the next pass starts with), and the logits of the steps with the hook
    installed."""
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


def _scaled(W, name, factor):
    W[name] = (W[name].float() * factor).to(torch.bfloat16)


CHANGES = {     # tensor or constant -> what becomes of it
    "bigram": lambda c, W: _scaled(W, "bigram", 1.3),
    "first row": lambda c, W: W.update(bigram=torch.cat([W["bigram"][:-1], W["bigram"][-1:] * 2])),
    "mul_prev": lambda c, W: c["embedding"]["bigram"].update(mul_prev=18),
    "mul_cur": lambda c, W: c["embedding"]["bigram"].update(mul_cur=102),
    "step": lambda c, W: W.update({"loop.step": W["loop.step"].flip(0).contiguous()}),
    "norm2": lambda c, W: W.update({"l1.norm2": (W["l1.norm2"].float() + 0.5).to(torch.bfloat16)}),
    "q bias": lambda c, W: W.update({"l1.mix.q.b": W["l1.mix.q.b"].flip(0).contiguous()}),
    "k bias": lambda c, W: W.update({"l1.mix.k.b": W["l1.mix.k.b"].flip(0).contiguous()}),
    "v bias": lambda c, W: W.update({"l1.mix.v.b": W["l1.mix.v.b"].flip(0).contiguous()}),
    "q taps": lambda c, W: W.update({"l1.mix.q.conv": W["l1.mix.q.conv"].flip(1).contiguous()}),
    "k taps": lambda c, W: W.update({"l1.mix.k.conv": W["l1.mix.k.conv"].flip(1).contiguous()}),
    "v taps": lambda c, W: W.update({"l1.mix.v.conv": W["l1.mix.v.conv"].flip(1).contiguous()}),
    "scale": lambda c, W: c["layers"][1]["mixer"].update(scale=0.5),
    "rot.dims": lambda c, W: c["layers"][1]["mixer"]["rot"].update(dims=12),
    "base": lambda c, W: c["layers"][1]["mixer"]["rot"].update(base=3000.0),
    "factor": lambda c, W: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=30.0),
    "fast": lambda c, W: c["layers"][1]["mixer"]["rot"]["scaling"].update(fast=1.5),
    "slow": lambda c, W: c["layers"][1]["mixer"]["rot"]["scaling"].update(slow=6.0),
    "original": lambda c, W: c["layers"][1]["mixer"]["rot"]["scaling"].update(original=4096),
    "plain rotation": lambda c, W: c["layers"][0]["mixer"]["rot"].update(scaling=None),
    "latent factor": lambda c, W: c["layers"][3]["mixer"]["rot"]["scaling"].update(factor=20.0),
    "latent scale": lambda c, W: c["layers"][3]["mixer"].update(scale=0.6),
    "sink": lambda c, W: W.update({"l3.mix.sink": (W["l3.mix.sink"].float() + 1.0).to(torch.bfloat16)}),
    "latent gate": lambda c, W: W.update({"l3.mix.g": W["l3.mix.g"].flip(0).contiguous()}),
    "dkv.norm": lambda c, W: W.update({"l0.mix.dkv.norm": W["l0.mix.dkv.norm"].flip(0).contiguous()}),
    "final": lambda c, W: W.update({"final.norm": (W["final.norm"].float() + 0.5).to(torch.bfloat16)}),
    "cap": lambda c, W: c.update(logit_softcap=8.0),
    "no cap": lambda c, W: c.update(logit_softcap=None),
    "times": lambda c, W: (c["loop"].update(times=1), W.update({"loop.step": W["loop.step"][:1]})),
    "start": lambda c, W: c["loop"].update(start=2),
    "stop": lambda c, W: c["loop"].update(stop=5),
    "no loop": lambda c, W: c.update(loop=None),
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
    assert (want - base).abs().max() > 0.02
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
                                  [3, 5, 7, 9, 11, 13, 88], [16, 32, 48, 64, 80]])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_many_sizes(cuts, dtype):
    """Cuts at, before and after page borders (16 tokens), the work items of the convolution (16), key steps (32, 64), and
    portions shorter than the taps, down to two tokens."""
    import llm_decoder as ld
    config, W = _case("full")
    toks = _tokens(90, config["vocab"], 5)
    eng = ld.Engine(_model(config, W, dtype))
    _close(_feed(eng, "a", toks, cuts), _oracle("full", config, W, toks), dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[2, 4, 6, 8, 11, 14, 30], [1, 2, 3, 20, 22, 37], [7, 8, 9, 16, 18]])
def test_short_portions_under_eight_taps(cuts):
    """Portions of one to three tokens under a convolution of eight taps: the state slot keeps rows of several portions."""
    import llm_decoder as ld
    config, W = _case("odd")
    toks = _tokens(40, config["vocab"], 7)
    _close(_feed(ld.Engine(_model(config, W)), "a", toks, cuts), _oracle("odd", config, W, toks))


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
        _close(torch.cat(got[r], 0), alone.double().cpu(), dtype, tol=2e-4, bf16_tol=0.04)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_large_decode_batch(dtype):
    """80 sequences of unequal length decode two tokens side by side: enough (token, key/value head) pairs for the
    tensor-core kernel of decoded tokens."""
    import llm_decoder as ld
    config = R.make_config([R.attention_layer(heads=6, kv_heads=2, dim=16, taps=3), R.latent_layer(heads=3, dim=8, rot_dim=8, kv_rank=16),
                            R.attention_layer(heads=4, kv_heads=2, dim=40, vdim=24, rot_dims=8, ff=None)], width=64,
                           loop={"start": 0, "stop": 2, "times": 2})
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
    """A pool of 160 tokens and two slots serves six requests one after another and interleaved: freed pages and slots come
    back (dirty) and the next request must not see the keys, the convolution rows or the last token they held."""
    import llm_decoder as ld
    config, W = _case("full")
    model = _model(config, W, max_tokens=160, max_seqs=2)
    assert len(model.states._kv) == 2 * 3 + 2               # the three looped layers have a pool per pass
    assert len(model.states._tables) == 3                   # layers with one, two and three key/value heads share a page table each
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
@pytest.mark.parametrize("tile_size", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_page_borders_and_far_keys_long_sequence(tile_size, dtype):
    """300 tokens of sharp attention: prompts cut around page borders and key steps, then 40 decoded tokens."""
    import llm_decoder as ld
    config = R.make_config([R.attention_layer(heads=4, kv_heads=1, dim=32, scale=0.8, rot_dims=8), R.latent_layer(heads=4, dim=16, rot_dim=8, scale=0.6)],
                           width=64, vocab=80)
    W = R.random_weights(config, 7)
    toks = _tokens(300, config["vocab"], 8)
    want = _oracle("edges", config, W, toks)
    eng = ld.Engine(_model(config, W, dtype, tile_size=tile_size))
    cuts = [5, 6, 63, 64, 65, 75, 77, 127, 129, 135, 192, 255, 256] + list(range(260, 300))
    _close(_feed(eng, "a", toks, cuts), want, dtype)
    eng.finish("a")
    _close(_feed(eng, "b", toks, [5, 290]), want, dtype)


def _needle_model(kind):
    """One layer of one head whose key map got a rank-one term: the needle token's key lands on the probe token's query, in
    the dimensions the rotation leaves alone, so the needle takes almost all the weight of the probe wherever it is.  The term
    reads a direction in which only the needle token has a component; pairs of tokens play no part (no pair embedding, a
    convolution of the token's own row)."""
    p, needle, probe = "l0.mix.", 7, 11
    if kind == "attention":
        config = R.make_config([R.attention_layer(heads=1, kv_heads=1, dim=24, vdim=16, taps=3, rot_dims=4, scale=1.5, ff=None)], width=64, vocab=40)
    else:
        config = R.make_config([R.latent_layer(heads=1, dim=20, rot_dim=4, kv_rank=48, scale=1.0, ff=None)], width=64, vocab=40)
    W = R.random_weights(config, 9)
    W["bigram"] = torch.zeros_like(W["bigram"])
    D = {k: v.double() for k, v in W.items()}
    eps, c = config["norm"]["eps"], config["layers"][0]["mixer"]
    every = R.norm1p(D["embed"], D["l0.norm1"], eps)
    if kind == "attention":
        own = torch.tensor([0.0, 0.0, 1.0]).to(torch.bfloat16)
        for n in "qkv":
            W[p + n + ".conv"] = own.expand(W[p + n].shape[0], 3).contiguous()
        W[p + "k.b"] = torch.zeros_like(W[p + "k.b"])
        q = D[p + "q"] @ every[probe] + D[p + "q.b"]
        q[:4] = 0.0
        W[p + "k"] = (D[p + "k"] * 0.3 + 60.0 * torch.outer(q / (q @ q), torch.linalg.pinv(every)[:, needle])).to(torch.bfloat16)
    else:
        q = (D[p + "q"] @ every[probe])[:c["dim"]]
        lat = R.rms(every @ D[p + "dkv"].T[:, :c["kv_rank"]], eps) * D[p + "dkv.norm"]
        W[p + "uk"] = (D[p + "uk"] * 0.1 + 18.0 * torch.outer(q / (q @ q), torch.linalg.pinv(lat)[:, needle])).to(torch.bfloat16)
        W[p + "sink"] = torch.full((1,), 4.0, dtype=torch.bfloat16)
    return config, W, needle, probe


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["attention", "latent"])
@pytest.mark.parametrize("where", [0, 1, 15, 16, 31, 32, 140, 399])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_far_key_among_hundreds(kind, where, dtype):
    """400 tokens: one key takes the probe's weight, from the first position to the neighbour; without it the logits differ.  The
    probe comes at the end of a prompt portion, or decoded alone."""
    import llm_decoder as ld
    config, W, needle, probe = _needle_model(kind)
    others = [t for t in range(40) if t not in (needle, probe)]
    rnd = random.Random(where)
    toks = [rnd.choice(others) for _ in range(400)] + [probe]
    without = R.forward(config, W, toks)[-1]
    toks[where] = needle
    want = R.forward(config, W, toks)
    assert (want[-1] - without).abs().max() > 0.5
    for cuts in ([400], [390], [where + 1, 399, 400]):
        _close(_feed(ld.Engine(_model(config, W, dtype)), "a", toks, cuts), want, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("shift", [-40.0, 0.0, 12.0, 60.0])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_from_nothing_to_everything(shift, dtype):
    """Sinks far below every score (an ordinary softmax), among them, and far above (the heads give next to nothing)."""
    import llm_decoder as ld
    config, W = _case("latent", seed=5)
    W["l0.mix.sink"] = (W["l0.mix.sink"].float() + shift).to(torch.bfloat16)
    toks = _tokens(600, config["vocab"], 17)
    want = R.forward(config, W, toks)
    _close(_feed(ld.Engine(_model(config, W, dtype)), "a", toks, [520] + list(range(570, 600))), want, dtype)


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
    """A 560-token portion followed by 150 decoded tokens (keys split over CTAs); the same request again cut at 300."""
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
def test_greedy_generation_through_the_scheduler(dtype):
    """Scheduler: five prompts of unequal length on four slots with a small token budget (chunked prompts, continuous
    batching, slot reuse); greedy tokens equal the oracle's argmax at every step (float32), and stay near its maximum
    (bfloat16)."""
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
                assert float(logits[t].max() - logits[t, o[t + 1]]) < 1.0


def _random_config(rnd):
    """Layer count and order, the loop, every size and constant drawn at random."""
    layers = []
    for _ in range(rnd.randint(2, 6)):
        ff = rnd.choice([None, 8, 30, 64, 100])
        sc = rnd.choice([None, R.scaling(rnd.choice([2.0, 8.0]), rnd.choice([16, 100, 1000]), rnd.choice([4.0, 32.0]), rnd.choice([0.5, 1.0]))])
        base = rnd.choice([50.0, 10000.0, 500000.0])
        if rnd.random() < 0.5:
            kv, dim = rnd.choice([1, 2, 3]), rnd.choice([8, 12, 16, 24, 33, 64])
            layers.append(R.attention_layer(heads=kv * rnd.randint(1, 4), kv_heads=kv, dim=dim, vdim=rnd.choice([dim, 8, 20, 72, 13]),
                                            taps=rnd.randint(1, 6), rot_dims=rnd.randrange(2, dim + 1, 2), base=base, sc=sc,
                                            scale=rnd.uniform(0.1, 0.6), ff=ff))
        else:
            layers.append(R.latent_layer(heads=rnd.randint(1, 9), dim=rnd.choice([8, 12, 16, 24, 20]), rot_dim=rnd.choice([2, 4, 8, 16, 40]),
                                         vdim=rnd.choice([8, 16, 40, 20, 6]), kv_rank=rnd.choice([8, 16, 20, 64, 72]), base=base, sc=sc,
                                         scale=rnd.uniform(0.1, 0.4), ff=ff))
    a = rnd.randrange(len(layers))
    loop = rnd.choice([None, {"start": a, "stop": rnd.randint(a + 1, len(layers)), "times": rnd.randint(1, 3)}])
    return R.make_config(layers, width=rnd.choice([40, 64, 72, 96, 50, 51]), vocab=rnd.choice([61, 97, 128]), loop=loop,
                         eps=rnd.choice([1e-5, 1e-6, 1e-3]), buckets=rnd.choice([1, 7, 101, 256]), mul_prev=rnd.randint(1, 10 ** 6),
                         mul_cur=rnd.randint(1, 10 ** 9), cap=rnd.choice([None, 10.0, 30.0]))


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
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot_dims,norm", [(4, 2, 16, 24, 6, 1), (3, 1, 7, 10, 4, 1), (2, 2, 64, 64, 64, 0), (6, 3, 128, 96, 32, 1),
                                                                   (2, 1, 130, 258, 2, 1), (5, 5, 8, 6, 0, 0), (1, 1, 512, 40, 512, 1)])
@pytest.mark.parametrize("taps", [0, 1, 2, 4, 7, 8])
def test_convolution_rotation_norm_append_alone(heads, kv_heads, dim, vdim, rot_dims, norm, taps):
    """pa_conv_rope_norm_append against the mechanisms one by one: three sequences through four steps (portions of one to 40
    tokens, cut into items of 8), queries, pool rows (read back through the page table) and the rows kept for the next step; and
    a layer without a pool."""
    from llm_decoder import _cabi
    from llm_decoder.seq_state import SequenceStateCache
    lib, dev, base, eps = _cabi.lib(), torch.device("cuda"), 300.0, 1e-5
    g = torch.Generator().manual_seed(dim + taps)
    steps = [[(0, 14), (1, 1), (2, 40)], [(2, 1), (0, 5)], [(1, 2), (0, 1), (2, 3)], [(0, 18), (1, 9)]]
    qc, kc, vc = heads * dim, kv_heads * dim, kv_heads * vdim
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1.2e-2)):
        e = 4 if dtype == torch.float32 else 2
        for own in (True, False):
            channels = qc + (kc + vc if own else 0)
            w = torch.randn(channels, taps, generator=g).mul(0.6).float() if taps else None
            wt = w.flip(1).t().contiguous().to(dev) if taps else None
            states = SequenceStateCache(3, 512, 16, dev)
            kv = states.add_kv_layer(kv_heads, dim, vdim, "f32" if e == 4 else "bf16")
            cst = states.add_state((taps - 1) * channels) if taps > 1 else None
            for t in states._states:
                t.fill_(9.0)                            # what a slot held before it is handed out
            slots = [states.alloc() for _ in range(3)]
            fed = [torch.zeros(0, channels, dtype=torch.float64) for _ in range(3)]
            turn = lambda x, t: R.turn_neighbours(x, t, {"dims": rot_dims, "base": base, "scaling": R.scaling()})  # noqa: E731
            for step in steps:
                batch = states.make_batch([(slots[i], [0] * n) for i, n in step])
                rows = batch.rows
                src = torch.randn(rows, channels + 4, generator=g).to(dtype)
                rope = None
                if rot_dims:
                    f, mult = R.stretched_frequencies(rot_dims, base, R.scaling())
                    rope = torch.empty(rows, rot_dims // 2, 2, device=dev)
                    fd = torch.tensor(f, dtype=torch.float64, device=dev)
                    assert lib.pa_rope_table_scaled(batch.row_pos.data_ptr(), rows, rot_dims, fd.data_ptr(), mult, rope.data_ptr(), _cabi.stream()) == 0
                x, q = src.to(dev), torch.zeros(rows, qc, dtype=dtype, device=dev)
                items, n = batch.portion_items(8)
                pt = kv.page_table_
                rc = lib.pa_conv_rope_norm_append(
                    x.data_ptr(), x.stride(0), 2, heads, kv_heads, dim, vdim, taps, _cabi.ptr(wt), _cabi.ptr(cst), rot_dims, _cabi.ptr(rope),
                    norm, eps, q.data_ptr(), qc, kv.key_buffer_.data_ptr() if own else None, kv.value_buffer_.data_ptr() if own else None,
                    pt.device_data().data_ptr(), pt.num_beams_, pt.num_tiles_, kv.total_pages_, kv.tile_size_, items.data_ptr(), n, 8, e,
                    _cabi.stream())
                assert rc == 0
                assert torch.equal(x.cpu(), src)
                got = q.double().cpu()
                table = pt.device_data().cpu().reshape(pt.num_beams_, kv_heads, pt.num_tiles_)
                kb, vb = kv.key_buffer_.double().cpu().reshape(-1, 16, dim), kv.value_buffer_.double().cpu().reshape(-1, 16, vdim)
                r0 = 0
                for i, cnt in step:
                    p0 = fed[i].shape[0]
                    fed[i] = torch.cat([fed[i], src[r0:r0 + cnt, 2:2 + channels].double()])
                    y = R.short_convolution(fed[i], w.double())[p0:] if taps else fed[i][p0:]
                    for t in range(cnt):
                        def head(a, pos=p0 + t, row=y[t]):
                            z = turn(row[a:a + dim], pos) if rot_dims else row[a:a + dim]
                            return R.rms(z, eps) if norm else z
                        for h in range(heads):
                            want = head(h * dim)
                            assert (got[r0 + t, h * dim:(h + 1) * dim] - want).abs().max() < tol * max(1.0, want.abs().max().item())
                        for gi in range(kv_heads if own else 0):
                            page, at = int(table[slots[i], gi, (p0 + t) // 16]), (p0 + t) % 16
                            want = head(qc + gi * dim)
                            assert (kb[page, at] - want).abs().max() < tol * max(1.0, want.abs().max().item())
                            want = y[t, qc + kc + gi * vdim:qc + kc + (gi + 1) * vdim]
                            assert (vb[page, at] - want).abs().max() < tol * max(1.0, want.abs().max().item())
                    r0 += cnt
                if cst is not None:
                    for i in range(3):
                        if fed[i].shape[0]:
                            want = torch.cat([torch.zeros(taps - 1, channels, dtype=torch.float64), fed[i]])[-(taps - 1):]
                            assert torch.equal(cst[slots[i]].double().cpu().reshape(taps - 1, channels), want)


@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv_rank,rot_dim", [(3, 16, 8), (16, 64, 32), (8, 136, 16), (5, 13, 6), (70, 24, 8), (20, 256, 64)])
@pytest.mark.parametrize("sink", [-50.0, 0.0, 3.0, 80.0, None])
def test_latent_attention_with_sinks_alone(heads, kv_rank, rot_dim, sink):
    """pa_latent_attention_sink over a paged pool: the float kernel, both tensor-core forms, with and without split keys, sinks
    from far below to far above the scores, against attention written out in float64."""
    from llm_decoder import _cabi
    from llm_decoder.seq_state import SequenceStateCache
    lib, dev, scale = _cabi.lib(), torch.device("cuda"), 0.3
    g = torch.Generator().manual_seed(heads + kv_rank)
    ctx, new, kd = [70, 0, 530], [40, 2, 1], kv_rank + rot_dim
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 2e-2)):
        e = 4 if dtype == torch.float32 else 2
        states = SequenceStateCache(3, 1024, 16, dev)
        kv = states.add_kv_layer(1, kd, 0, "f32" if e == 4 else "bf16")
        slots = [states.alloc() for _ in range(3)]
        for sl, n in zip(slots, ctx):
            if n:
                states.extend(sl, n)
        batch = states.make_batch([(sl, [0] * n) for sl, n in zip(slots, new)])
        rows = batch.rows
        pool = torch.randn(kv.key_buffer_.numel() // kd, kd, generator=g).to(dtype)
        kv.key_buffer_.view(-1, kd).copy_(pool)
        pt = kv.page_table_
        table = pt.device_data()
        tab = table.cpu().reshape(pt.num_beams_, pt.num_tiles_)
        ql, qr = torch.randn(heads, rows, kv_rank, generator=g).to(dtype), torch.randn(rows, heads * rot_dim, generator=g).to(dtype)
        sk = None if sink is None else torch.randn(heads, generator=g) + sink
        want, r = torch.zeros(heads, rows, kv_rank, dtype=torch.float64), 0
        for sl, c0, n in zip(slots, ctx, new):
            keys = torch.stack([pool[int(tab[sl, j // 16]) * 16 + j % 16] for j in range(c0 + n)]).double()
            for t in range(n):
                k = keys[:c0 + t + 1]
                s = torch.cat([ql[:, r].double(), qr[r].double().reshape(heads, rot_dim)], 1) @ k.T * scale
                if sk is not None:
                    s = torch.cat([s, sk.double()[:, None]], 1)
                want[:, r] = torch.softmax(s, -1)[:, :k.shape[0]] @ k[:, :kv_rank]
                r += 1
        qld, qrd, skd = ql.to(dev), qr.to(dev), None if sk is None else sk.to(dev)
        forms = [(0, lib.pa_latent_attention_tile_tokens(heads))]
        mt = lib.pa_latent_attention_mma_tile_tokens(heads, kv_rank, rot_dim, e)
        forms += [(2, mt)] if mt else []
        for form, tokens in forms:
            for nsplit in (1, 3):
                out = torch.zeros(heads, rows, kv_rank, dtype=dtype, device=dev)
                for kind, group in batch.query_tiles(tokens).items():
                    if group is None:
                        continue
                    tiles, ntiles, _longest = group
                    ws = torch.empty(max(1, lib.pa_latent_attention_workspace_bytes(ntiles, heads, kv_rank, nsplit)), dtype=torch.uint8, device=dev)
                    rc = lib.pa_latent_attention_sink(qld.data_ptr(), kv_rank, rows * kv_rank, qrd.data_ptr(), heads * rot_dim, rot_dim,
                                                      kv.key_buffer_.data_ptr(), table.data_ptr(), pt.num_beams_, pt.num_tiles_, kv.total_pages_, 16,
                                                      tiles.data_ptr(), ntiles, heads, kv_rank, rot_dim, scale, _cabi.ptr(skd), out.data_ptr(),
                                                      kv_rank, rows * kv_rank, e, nsplit, (3 if kind == 1 else 2) if form else 0, ws.data_ptr(),
                                                      ws.numel(), _cabi.stream())
                    assert rc == 0
                err = (out.double().cpu() - want).abs().max().item()
                assert err < tol * max(1.0, want.abs().max().item()), (dtype, form, nsplit, err)


@pytest.mark.gpu
@pytest.mark.parametrize("kv_rank,rot_dim,dims,heads", [(40, 16, 16, 3), (13, 6, 4, 5), (72, 2, 2, 1), (16, 4, 0, 2)])
def test_latent_append_with_query_rotation_alone(kv_rank, rot_dim, dims, heads):
    """pa_latent_turn_append: pool rows (norm with a gain, shared key part rotated) and the queries of the same rows rotated in
    place, at positions around page borders, with a stretched rotation."""
    from llm_decoder import _cabi
    from llm_decoder.seq_state import SequenceStateCache
    lib, dev, eps, plain = _cabi.lib(), torch.device("cuda"), 1e-5, 7
    g = torch.Generator().manual_seed(kv_rank)
    ctx, new = [14, 0, 1000], [5, 1, 20]
    rows, pos = sum(new), [p for c, n in zip(ctx, new) for p in range(c, c + n)]
    rot = {"dims": dims, "base": 300.0, "scaling": R.scaling(4.0, 32, 2.0, 0.5)}
    turn = lambda v, p: R.turn_neighbours(v, p, rot) if dims else v  # noqa: E731
    for dtype, tol in ((torch.float32, 4e-5), (torch.bfloat16, 5e-2)):
        e = 4 if dtype == torch.float32 else 2
        states = SequenceStateCache(3, 2048, 16, dev)
        kv = states.add_kv_layer(1, kv_rank + rot_dim, 0, "f32" if e == 4 else "bf16")
        slots = [states.alloc() for _ in range(3)]
        for sl, n in zip(slots, ctx):
            if n:
                states.extend(sl, n)
        batch = states.make_batch([(sl, [0] * n) for sl, n in zip(slots, new)])
        qd = plain + rot_dim
        x = torch.randn(rows, heads * qd + kv_rank + rot_dim + 3, generator=g).to(dtype)
        gain = torch.rand(kv_rank, generator=g) + 0.5
        rope = torch.empty(rows, max(1, dims // 2), 2, device=dev)
        if dims:
            f, mult = R.stretched_frequencies(dims, 300.0, rot["scaling"])
            fd = torch.tensor(f, dtype=torch.float64, device=dev)
            assert lib.pa_rope_table_scaled(batch.row_pos.data_ptr(), rows, dims, fd.data_ptr(), mult, rope.data_ptr(), _cabi.stream()) == 0
            want = torch.tensor([[[math.cos(p * fi) * mult, math.sin(p * fi) * mult] for fi in f] for p in pos])
            assert (rope.cpu() - want).abs().max() < 1e-6
        X, gd, pt = x.to(dev), gain.to(dev), kv.page_table_
        table = pt.device_data()
        assert lib.pa_latent_turn_append(kv.key_buffer_.data_ptr(), table.data_ptr(), pt.num_beams_, pt.num_tiles_, kv.total_pages_, 16, kv_rank,
                                         rot_dim, dims, 0, X.data_ptr(), X.stride(0), heads * qd, gd.data_ptr(), eps, rope.data_ptr(), X.data_ptr(),
                                         X.stride(0), plain, heads, qd, batch.row_slot.data_ptr(), batch.row_pos.data_ptr(), rows, e,
                                         _cabi.stream()) == 0
        xd, got = x.double(), X.double().cpu()
        pool, tab = kv.key_buffer_.double().cpu().reshape(-1, 16, kv_rank + rot_dim), table.cpu().reshape(pt.num_beams_, pt.num_tiles_)
        slot_of = [sl for sl, n in zip(slots, new) for _ in range(n)]
        for r in range(rows):
            row = pool[int(tab[slot_of[r], pos[r] // 16]), pos[r] % 16]
            c0 = heads * qd
            assert (row[:kv_rank] - R.rms(xd[r, c0:c0 + kv_rank], eps) * gain.double()).abs().max() < tol
            assert (row[kv_rank:] - turn(xd[r, c0 + kv_rank:c0 + kv_rank + rot_dim], pos[r])).abs().max() < tol
            want = xd[r].clone()
            for h in range(heads):
                a = h * qd + plain
                want[a:a + rot_dim] = turn(want[a:a + rot_dim], pos[r])
            assert (got[r] - want).abs().max() < tol


@pytest.mark.gpu
@pytest.mark.parametrize("width", [64, 51, 2000])
def test_pair_embedding_alone(width):
    """pa_embedding_bigram against the rows written out: first tokens, ids outside the vocabulary (zeros), factors whose
    products leave 32 bits, factors below zero, a second copy."""
    from llm_decoder import _cabi
    lib, dev, vocab, buckets = _cabi.lib(), torch.device("cuda"), 70000, 101
    g = torch.Generator().manual_seed(width)
    emb, pairs = torch.randn(vocab, width, generator=g), torch.randn(buckets + 1, width, generator=g)
    ids = [0, 5, vocab - 1, 69000, 3, -1, vocab]
    prev = [-1, 0, vocab - 1, -1, 68000, 5, 5]
    for mp, mc in ((31, 5), (10 ** 12 + 39, 2 ** 33 + 1), (-7, 3)):
        for dtype in (torch.float32, torch.bfloat16):
            E, B = emb.to(dtype), pairs.to(dtype)
            want = torch.stack([E[i].float() * 2.0 + B[buckets if p == -1 else (p * mp + i * mc) % buckets].float() if 0 <= i < vocab
                                else torch.zeros(width) for i, p in zip(ids, prev)])
            i32 = dict(dtype=torch.int32, device=dev)
            Ed, Bd, idd, pd = E.to(dev), B.to(dev), torch.tensor(ids, **i32), torch.tensor(prev, **i32)
            out, copy = torch.empty(7, width, device=dev), torch.empty(7, width, device=dev)
            assert lib.pa_embedding_bigram(Ed.data_ptr(), Bd.data_ptr(), E.element_size(), idd.data_ptr(), pd.data_ptr(), 7, width, vocab, buckets,
                                           mp, mc, 2.0, out.data_ptr(), copy.data_ptr(), _cabi.stream()) == 0
            assert (out.cpu() - want).abs().max() < 1e-6 and torch.equal(out, copy)


@pytest.mark.gpu
@pytest.mark.parametrize("width", [64, 51, 2000])
@pytest.mark.parametrize("has", ["y y2 base step h1 h2", "y h1", "base step h1 h2", "y y2", "step h2", "h1 h2"])
def test_residual_add_and_two_norms_alone(width, has):
    from llm_decoder import _cabi
    lib, dev, rows, eps = _cabi.lib(), torch.device("cuda"), 9, 1e-5
    g = torch.Generator().manual_seed(width)
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 1e-2)):
        x, base, step = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g), torch.randn(width, generator=g)
        y, y2 = torch.randn(rows, width, generator=g).to(dtype), torch.randn(rows, width, generator=g).to(dtype)
        g1, g2 = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
        on = lambda t, n: t.to(dev) if n in has.split() else None  # noqa: E731
        xd, yd, y2d, bd, sd = x.to(dev), on(y, "y"), on(y2, "y2"), on(base, "base"), on(step, "step")
        h1, h2, g1d, g2d = on(torch.zeros_like(y), "h1"), on(torch.zeros_like(y), "h2"), g1.to(dev), g2.to(dev)
        assert lib.pa_residual_add_norm2_pass(xd.data_ptr(), rows, width, _cabi.ptr(yd), _cabi.ptr(y2d), None, None, None, 0, 0, None, _cabi.ptr(bd),
                                              _cabi.ptr(sd), eps, g1d.data_ptr(), _cabi.ptr(h1), g2d.data_ptr(), _cabi.ptr(h2), y.element_size(),
                                              _cabi.stream()) == 0
        want = x.double()
        for n, t in (("y", y), ("y2", y2), ("base", base), ("step", step)):
            want = want + t.double() if n in has.split() else want
        assert (xd.double().cpu() - want).abs().max() < 3e-6
        for h, gain in ((h1, g1), (h2, g2)):
            if h is not None:
                ref = R.rms(want, eps) * gain.double()
                assert (h.double().cpu() - ref).abs().max() < tol * max(1.0, ref.abs().max().item())


@pytest.mark.gpu
@pytest.mark.parametrize("cols,in_pad,gate_off", [(64, 0, 8), (51, 3, 5), (4096, 8, 16), (40, 4, 0)])
def test_element_gate_alone(cols, in_pad, gate_off):
    from llm_decoder import _cabi
    lib, dev, rows = _cabi.lib(), torch.device("cuda"), 7
    g = torch.Generator().manual_seed(cols)
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-2)):
        x, gate = torch.randn(rows, cols + in_pad, generator=g).to(dtype), torch.randn(rows, gate_off + cols + 8, generator=g).mul(3).to(dtype)
        want = x[:, :cols].double() / (1.0 + torch.exp(-gate[:, gate_off:gate_off + cols].double()))
        xd, gd = x.to(dev), gate.to(dev)
        out = torch.zeros(rows, cols, dtype=dtype, device=dev)
        e = x.element_size()
        for dst, stride in ((out, cols), (xd, cols + in_pad)):          # a place of its own, then in place
            assert lib.pa_gate_rows(xd.data_ptr(), cols + in_pad, gd.data_ptr() + gate_off * e, gd.stride(0), cols, rows, dst.data_ptr(), stride, e,
                                    _cabi.stream()) == 0
            assert (dst[:, :cols].double().cpu() - want).abs().max() < tol * want.abs().max().item()
        assert torch.equal(xd[:, cols:].cpu(), x[:, cols:])


# ---- configuration -------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
def test_configuration_errors():
    def broken(name, change):
        config, W = _case(name)
        config = json.loads(json.dumps(config))
        change(config)
        with pytest.raises(ValueError):
            _model(config, W)
    broken("attention", lambda c: c["layers"][0]["mixer"].update(heads=6))          # the tensors have other rows
    broken("attention", lambda c: c["layers"][0]["mixer"].update(conv=4))
    broken("attention", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26))
    broken("attention", lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0))
    broken("attention", lambda c: c["embedding"]["bigram"].update(buckets=88))
    broken("attention", lambda c: c["layers"][0].update(type="mamba2"))
    broken("latent", lambda c: c["layers"][0]["mixer"].update(kv_rank=8))
    broken("latent", lambda c: c["layers"][0]["mixer"].update(vdim=24))
    broken("latent", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7))
    broken("loop", lambda c: c["loop"].update(stop=4))
    broken("loop", lambda c: c["loop"].update(times=2))                             # a step vector per pass
    broken("full", lambda c: c["layers"][1]["mlp"].update(ff=8))
    broken("full", lambda c: c["layers"][1]["mlp"].update(kind="moe"))


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
