"""Rupulix (parallel residual streams; windowed latent attention with a rotated part and a sink; attention with mixed scores beside a
gated linear recurrence; a repeated span of layers) against the plain oracle of oracle/rupulix.py.

Small configurations with their own random weights; the oracle runs in float64.  The engine's "f32" precision is held to a tight
bar (a window one token off, a sink left out, a state of the wrong slot or pass, a head mixed with the wrong one shows), the serving
precision to the bar its operand rounding allows.
"""
import copy
import math

import numpy as np
import pytest
import torch

from oracle import rupulix as O

T64 = torch.float64


# ---------------------------------------------------------------------------------------------------- configurations
def latent(heads=5, dim=20, rot_dim=6, vdim=28, kv_rank=44, size=37, scale=0.2, base=10000.0, dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim if dims is None else dims}}
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m}


def recurrence(width=60, blocks=3, conv=4):
    return {"width": width, "blocks": blocks, "conv": conv}


def parallel(heads=6, kv_heads=2, dim=18, vdim=26, scale=0.25, base=5000.0, dims=None, left_scale=0.7, right_scale=1.2, right=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dim if dims is None else dims}}
    return {"type": "parallel", "mixer": {"left": left, "right": right or recurrence(), "left_scale": left_scale, "right_scale": right_scale}}


def layer(mx, ff=52):
    return dict(copy.deepcopy(mx), mlp={"kind": "dense", "ff": ff} if ff else None)


def config(layers, width=120, vocab=211, eps=1e-5, streams=3, logit_scale=0.6, loop=None):
    c = {"architecture": "Rupulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "logit_scale": logit_scale, "layers": copy.deepcopy(layers)}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# five layers of unequal geometry, both mixers at least twice, one layer without a feed-forward, the middle of the list run twice
FULL = config([layer(parallel()),
               layer(latent()),
               layer(parallel(heads=2, kv_heads=2, dim=16, vdim=8, dims=4, right=recurrence(36, 2, 3)), None),
               layer(latent(heads=3, dim=9, rot_dim=4, vdim=7, kv_rank=21, size=70, scale=0.3, base=300.0), 30),
               layer(parallel(heads=4, kv_heads=1, dim=10, vdim=40, scale=0.3, base=100.0, right=recurrence(34, 1, 2)), 64)], loop=(1, 4, 2))
SINGLE = {
    "latent_only": config([layer(latent(), None)]),
    "latent_one_head_window_one": config([layer(latent(heads=1, dim=16, rot_dim=2, vdim=16, kv_rank=8, size=1))], width=64, vocab=70, streams=2),
    "latent_no_window": config([layer(latent(size=0), None)], streams=1),
    "latent_window_longer_than_the_prompt": config([layer(latent(size=500))], streams=4),
    "latent_partly_rotated": config([layer(latent(rot_dim=12, dims=4))]),
    "latent_odd_widths": config([layer(latent(heads=3, dim=11, rot_dim=2, vdim=13, kv_rank=19, size=20), 33)], width=66, vocab=90, streams=5),
    "latent_wide_rank": config([layer(latent(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=300, size=50), None)], width=96),
    "parallel_only": config([layer(parallel(), None)]),
    "parallel_one_head": config([layer(parallel(heads=1, kv_heads=1, dim=16, vdim=12, right=recurrence(16, 1, 1)), 24)], width=64, vocab=70, streams=1),
    "parallel_every_head_its_own_keys": config([layer(parallel(heads=5, kv_heads=5, dim=8, vdim=24), None)], streams=2),
    "parallel_one_key_head_unrotated": config([layer(parallel(heads=4, kv_heads=1, dim=13, vdim=21, dims=0), None)], width=66, vocab=90),
    "parallel_wide_values": config([layer(parallel(heads=2, kv_heads=1, dim=12, vdim=300), None)], width=80),
    "parallel_keys_wider_than_the_tiles": config([layer(parallel(heads=6, kv_heads=6, dim=96, vdim=32, scale=0.1), None)], width=96),
    "recurrence_a_block_per_channel": config([layer(parallel(right=recurrence(24, 24, 4)))], width=72, vocab=90),
    "recurrence_long_convolution": config([layer(parallel(right=recurrence(40, 2, 7)))], logit_scale=1.0),
    "recurrence_wide_blocks": config([layer(parallel(right=recurrence(420, 2, 4)), None)], width=96, vocab=100),
    "recurrence_one_block": config([layer(parallel(right=recurrence(130, 1, 2)), 20)], streams=6),
    "a_repeated_layer": config([layer(latent(), 20), layer(parallel(), 40)], loop=(0, 2, 3), streams=2),
    "a_span_that_runs_once": config([layer(latent(), 20), layer(parallel(), 40)], loop=(1, 2, 1), streams=8),
}

F32_TOL, SPLIT_TOL = 2e-5, 2e-3


def tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def rel(a, b):
    a, b = np.asarray(a, np.float64), np.asarray(b, np.float64)
    return float(np.abs(a - b).max() / max(np.abs(b).max(), 1e-30))


def oracle_logits(cfg, w, ids, state=None):
    return O.forward(cfg, w, ids, state).numpy()


def bf(t):
    return t.to(torch.bfloat16).to(T64)


def sharp_model(seed, size=33, far=False):
    """Scores with a spread of several units (a query looks at one or two keys of what it sees, wherever they are), slow decays (the
    recurrence remembers hundreds of tokens), large sinks and strong mixing of heads: a key just inside or just outside a window, a sink
    that is left out, a state that was not carried moves the logits by O(1).  far: no window."""
    cfg = config([layer(latent(heads=4, dim=24, rot_dim=8, vdim=24, kv_rank=40, size=0 if far else size, scale=1.2, base=1e5), None),
                  layer(parallel(heads=4, kv_heads=2, dim=16, vdim=24, scale=1.1, base=1e5, right=recurrence(48, 2, 4)), 40),
                  layer(latent(heads=2, dim=16, rot_dim=16, vdim=32, kv_rank=32, size=0 if far else size + 8, scale=1.4, base=1e6), None),
                  layer(latent(heads=2, dim=32, rot_dim=4, vdim=16, kv_rank=24, size=0 if far else 64, scale=1.0))], width=128, vocab=200, streams=2, loop=(1, 3, 2))
    w = O.random_weights(cfg, seed)
    for k in w:
        if k.endswith("lam"):
            w[k] = bf(w[k] - 2.0)
        if k.endswith("sink"):
            w[k] = bf(w[k] + 4.0)
        if k.endswith("mix.q") or k.endswith("left.q") or k.endswith("left.k"):
            w[k] = bf(w[k] * 1.5)
        if k.endswith("q.norm") or k.endswith("k.norm"):
            w[k] = bf(w[k] * 1.2)
    return cfg, w


# ---------------------------------------------------------------------------------------------------- CPU: the oracle itself
def test_oracle_prefill_equals_token_by_token():
    w = O.random_weights(FULL, 1)
    ids = tokens(90, FULL["vocab"], 2)
    whole = oracle_logits(FULL, w, ids)
    s = O.State(FULL)
    step = np.concatenate([oracle_logits(FULL, w, ids[:3], s)] + [oracle_logits(FULL, w, [t], s) for t in ids[3:]])
    assert rel(step, whole) < 1e-9


def test_oracle_mechanisms_on_known_answers():
    t = lambda *v: torch.tensor(v, dtype=T64)
    assert torch.allclose(O.rms(t(3., 4.), 0.5), t(3., 4.) / math.sqrt(13.0))
    # rotation: neighbours turn together, or dimension i with dimension i + dims / 2; the rest passes
    x = t(1., 2., 0., 0., 9.)[None, None]
    y = O.rotate(x, torch.tensor([3]), 4, 100.0, True)[0, 0]
    assert torch.allclose(y, t(math.cos(3.), 2 * math.cos(.3), math.sin(3.), 2 * math.sin(.3), 9.))
    y = O.rotate(x, torch.tensor([3]), 2, 100.0, False)[0, 0]
    assert torch.allclose(y, t(math.cos(3.) - 2 * math.sin(3.), 2 * math.cos(3.) + math.sin(3.), 0., 0., 9.))
    # visibility, softmax with one more term in the denominator
    assert O.visible(9, 3).tolist() == [7, 8, 9] and O.visible(1, 3).tolist() == [0, 1] and O.visible(4, 1).tolist() == [4] and O.visible(2, 0).tolist() == [0, 1, 2]
    s = O.softmax_with_sink(torch.log(t(1., 2.))[None], torch.log(t(5.)))
    assert torch.allclose(s, t(1., 2.)[None] / 8.0) and torch.allclose(O.softmax_with_sink(torch.log(t(1., 3.))[None]), t(.25, .75)[None])
    # causal convolution: the last column weighs the current token, the bias joins the sum, the window carries the inputs before the portion
    cv, win = O.causal_conv(t(1., 2., 4.)[:, None], t(100., 10., 1.)[None], t(0.5), t(7., 8.)[:, None])
    assert cv[:, 0].tolist() == [781.5, 812.5, 124.5] and win[:, 0].tolist() == [2., 4.]
    # equal parts of a row under square matrices [out, in]
    w = torch.stack([torch.tensor([[1., 2.], [0., 1.]], dtype=T64), torch.tensor([[0., 1.], [3., 0.]], dtype=T64)])
    assert O.block_linear(t(1., 10., 5., 7.)[None], w, torch.tensor([[0., 1.], [2., 0.]], dtype=T64)).tolist() == [[21., 11., 9., 15.]]
    # linear recurrence: the input is scaled so that a unit-variance input keeps the state's variance
    S, last = O.linear_recurrence(torch.log(t(0.6, 0.8))[:, None], t(1., 10.)[:, None], t(2.))
    assert torch.allclose(S[:, 0], t(0.6 * 2 + 0.8, 0.8 * 2.0 + 6.0)) and torch.allclose(last, S[1])
    assert torch.allclose(O.softplus(t(0., 50., -50.)), t(math.log(2.), 50., math.exp(-50.)))
    # streams: weighted sum in; all streams at once out, the table indexed [from, to]
    xs = t(1., 10.)[:, None, None]
    assert O.stream_in(xs, t(2., 3.)).item() == 32.0
    assert O.stream_out(xs, torch.tensor([[1., 5.], [0., 2.]], dtype=T64), t(1., -1.), t(100.)[None])[:, 0, 0].tolist() == [101., -75.]
    p = {"up": torch.eye(2, dtype=T64), "down": torch.tensor([[1., 1.], [0., 2.]], dtype=T64)}
    assert O.feed_forward(t(3., -2.)[None], p, "").tolist() == [[9., 0.]]
    assert torch.allclose(O.gelu_tanh(t(1.3, -0.7)), torch.nn.functional.gelu(t(1.3, -0.7), approximate="tanh"))
    assert O.run_order({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3, 4] and O.run_order({"layers": [0] * 2}) == [0, 1]


def test_oracle_sees_what_the_sharp_tests_are_about():
    cfg, w = sharp_model(41)
    ids = tokens(200, cfg["vocab"], 42)
    base = oracle_logits(cfg, w, ids)
    for li in (0, 2, 3):
        for by in (1, -1):
            other = copy.deepcopy(cfg)
            other["layers"][li]["mixer"]["mask"]["size"] += by
            assert rel(oracle_logits(other, w, ids)[80:], base[80:]) > 5e-3, (li, by)
        no_sink = dict(w)
        no_sink[f"l{li}.mix.sink"] = torch.full_like(w[f"l{li}.mix.sink"], -1e30)
        assert rel(oracle_logits(cfg, no_sink, ids), base) > 1e-2
    for name, swap in (("l1.mix.left.talk", lambda t: t.T), ("l1.mix.left.talk", lambda t: torch.eye(4, dtype=T64)), ("l1.hc1.mix", lambda t: t.T), ("l2.hc1.in", lambda t: t.flip(0))):
        assert rel(oracle_logits(cfg, dict(w, **{name: swap(w[name])}), ids), base) > 1e-2, name
    for ri in (1, 3):                                                # either pass: a state or the convolution's inputs not carried over a cut, or taken from the other pass
        lost = O.State(cfg)
        oracle_logits(cfg, w, ids[:120], lost)
        lost.mem[ri] = torch.zeros_like(lost.mem[ri])
        assert rel(oracle_logits(cfg, w, ids[120:], lost), base[120:]) > 1e-2
        lost = O.State(cfg)
        oracle_logits(cfg, w, ids[:120], lost)
        lost.win[ri] = torch.zeros_like(lost.win[ri])
        assert rel(oracle_logits(cfg, w, ids[120:], lost), base[120:]) > 1e-2
    for part in ("mem", "win", "rows"):
        lost = O.State(cfg)
        oracle_logits(cfg, w, ids[:120], lost)
        a = getattr(lost, part)
        a[1], a[3] = a[3], a[1]
        assert rel(oracle_logits(cfg, w, ids[120:], lost), base[120:]) > 1e-2, part
    cfg, w = sharp_model(43, far=True)                                # no window: single keys hundreds of tokens back carry the output
    ids = tokens(400, cfg["vocab"], 44)
    base = oracle_logits(cfg, w, ids)
    near = copy.deepcopy(cfg)
    near["layers"][0]["mixer"]["mask"] = {"size": 200}
    assert rel(oracle_logits(near, w, ids)[300:], base[300:]) > 1e-2


# dim, rotated dimensions, vdim, rank, window of latent attention; dim, key heads, vdim of the other: widths below, at and above the tensor-core tiles' own
TENSOR_CORE_SHAPES = [(48, 16, 64, 64, 40, 32, 2, 64), (56, 16, 48, 96, 65, 48, 2, 128), (96, 32, 128, 72, 33, 64, 3, 136), (128, 40, 96, 128, 100, 120, 2, 192),
                      (120, 2, 200, 160, 31, 40, 1, 20), (192, 64, 256, 192, 64, 128, 2, 256), (300, 20, 128, 64, 50, 128, 4, 192), (256, 128, 256, 64, 40, 100, 3, 248)]


def sharp_attention(dim, rot_dim, vdim, rank, size, ldim, groups, lvdim):
    cfg = config([layer(latent(heads=3, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, size=size, scale=3.0 / math.sqrt(dim), base=1e5), None),
                  layer(parallel(heads=2 * groups, kv_heads=groups, dim=ldim, vdim=lvdim, scale=2.0 / math.sqrt(ldim), base=1e5, dims=ldim // 2, left_scale=1.5,
                                 right=recurrence(96, 2, 4)), None)], width=128, vocab=150, streams=2)
    w = O.random_weights(cfg, 45)
    w["l0.mix.q"] = bf(w["l0.mix.q"] * 1.5)
    w["l0.mix.sink"] = bf(w["l0.mix.sink"] + 2.0)
    return cfg, w, tokens(260, cfg["vocab"], 46)


@pytest.mark.parametrize("shape", TENSOR_CORE_SHAPES)
def test_oracle_sees_the_edges_of_the_tensor_core_tests(shape):
    cfg, w, ids = sharp_attention(*shape)
    want = oracle_logits(cfg, w, ids)
    for by in (1, -1):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] += by
        assert rel(oracle_logits(other, w, ids)[150:], want[150:]) > 5 * SPLIT_TOL, by
    assert rel(oracle_logits(cfg, dict(w, **{"l1.mix.left.talk": w["l1.mix.left.talk"].T}), ids), want) > 5 * SPLIT_TOL


# ---------------------------------------------------------------------------------------------------- GPU
def make(cfg, seed=0, weights=None, **opts):
    import crane_b200
    w = weights or O.random_weights(cfg, seed)
    opts.setdefault("max_tokens", 1024)
    opts.setdefault("max_batch", 4)
    m = crane_b200.RupulixModel(cfg, device=0, **opts)
    m.load_checkpoint((k, t.to(torch.float32).numpy()) for k, t in w.items())
    return m, w


def all_rows(n):
    return list(range(n))


@pytest.mark.gpu
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(name):
    cfg = SINGLE[name]
    for precision, tol in (("f32", F32_TOL), ("split", SPLIT_TOL)):
        m, w = make(cfg, 3, precision=precision)
        ids = tokens(100, cfg["vocab"], 4)
        want = oracle_logits(cfg, w, ids)
        assert rel(m.step_batch([(0, ids, all_rows(100))]), want) < tol
        m.clear_kv_cache()
        rows = [m.step_batch([(0, ids[:2], [0, 1])])] + [m.step_batch([(0, [t], [0])]) for t in ids[2:70]]
        assert rel(np.concatenate(rows), want[:70]) < tol
        m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("precision,tol", [("f32", F32_TOL), ("split", SPLIT_TOL)])
def test_whole_model_prefill_and_token_by_token_decoding(precision, tol):
    m, w = make(FULL, 5, precision=precision)
    ids = tokens(170, FULL["vocab"], 6)
    want = oracle_logits(FULL, w, ids)
    got = m.step_batch([(0, ids, all_rows(len(ids)))])
    assert rel(got, want) < tol
    m.clear_kv_cache()
    rows = [m.step_batch([(0, ids[:3], [0, 1, 2])])]
    rows += [m.step_batch([(0, [t], [0])]) for t in ids[3:]]       # long decoding through two page borders, every window passed, every state carried 167 times
    step = np.concatenate(rows)
    assert rel(step, want) < tol
    if precision == "f32":
        assert rel(step, got) < 1e-5
    m.close()


@pytest.mark.gpu
def test_plain_bf16_precision_is_close():
    m, w = make(FULL, 7, precision="bf16")
    ids = tokens(90, FULL["vocab"], 8)
    got, want = m.step_batch([(0, ids, all_rows(90))]), oracle_logits(FULL, w, ids)
    assert rel(got, want) < 6e-2
    m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[2, 2, 2, 61, 3, 64, 1, 1, 30, 2], [63, 1, 1, 63, 2, 36], [1] * 5 + [95, 66], [31, 33, 32, 64, 6], [17, 18, 19, 112]])
def test_portions_of_any_size_match_the_whole_prompt(cuts):
    n = sum(cuts)
    ids = tokens(n, FULL["vocab"], 10)
    for precision, tol in (("f32", F32_TOL), ("split", SPLIT_TOL)):
        m, w = make(FULL, 9, precision=precision)
        at, rows = 0, []
        for c in cuts:
            rows.append(m.step_batch([(0, ids[at:at + c], all_rows(c))]))
            at += c
        assert rel(np.concatenate(rows), oracle_logits(FULL, w, ids)) < tol
        m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("precision,tol", [("f32", F32_TOL), ("split", SPLIT_TOL)])
def test_unequal_requests_in_one_batch_match_each_alone(precision, tol):
    m, w = make(FULL, 11, precision=precision, max_tokens=1024)
    lens = [97, 5, 130, 64]
    prompts = [tokens(n, FULL["vocab"], 20 + i) for i, n in enumerate(lens)]
    want = [oracle_logits(FULL, w, p) for p in prompts]
    seqs = [0] + [m.seq_create() for _ in range(3)]
    got = [[] for _ in lens]
    at = [0] * 4
    # a different mixture every step: portions of some beside single tokens of others, one request sitting a step out
    plan = [[(0, 40), (1, 2), (2, 1)], [(2, 64), (3, 63), (0, 1)], [(1, 1), (3, 1), (0, 56), (2, 2)], [(1, 2), (2, 63)]]
    for stepn in plan:
        entries = [(seqs[i], prompts[i][at[i]:at[i] + c], all_rows(c)) for i, c in stepn]
        lg = m.step_batch(entries)
        r = 0
        for i, c in stepn:
            got[i].append(lg[r:r + c]); r += c; at[i] += c
    for i in range(4):
        g = np.concatenate(got[i])
        assert rel(g, want[i][:len(g)]) < tol, i
    m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("precision,tol", [("f32", F32_TOL), ("split", SPLIT_TOL)])
def test_sequences_decoded_side_by_side_match_each_alone(precision, tol):
    m, w = make(FULL, 12, precision=precision, max_tokens=1024)
    prompts = [tokens(n + 20, FULL["vocab"], 60 + n) for n in (1, 64, 31, 40)]
    want = [oracle_logits(FULL, w, p) for p in prompts]
    seqs = [0] + [m.seq_create() for _ in range(3)]
    for s, p in zip(seqs, prompts):
        m.step_batch([(s, p[:-20], [])])
    for t in range(20):                                          # one, two, three, four rows in turn; a sequence that sits out keeps its state
        live = [i for i in range(4) if t < 4 or (t + i) % 4 != 0]
        if t == 3:
            live = [2]
        at = [m.seq_len(s) for s in seqs]
        lg = m.step_batch([(seqs[i], [prompts[i][at[i]]], [0]) for i in live])
        for r, i in enumerate(live):
            assert rel(lg[r], want[i][at[i]]) < tol, (t, i)
    m.close()


@pytest.mark.gpu
def test_many_sequences_decoded_side_by_side():
    # more rows than the weight-streaming linears take, then more than the key splits do: single tokens through the many-row kernels
    cfg = config([layer(latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=24, size=20), 40), layer(parallel(heads=2, kv_heads=1, dim=16, vdim=16, right=recurrence(32, 2, 4)))], width=64, vocab=90)
    w = O.random_weights(cfg, 61)
    prompts = [tokens(9 + 3 * i, cfg["vocab"], 70 + i) for i in range(22)]
    want = [oracle_logits(cfg, w, p) for p in prompts]
    for precision, tol in (("f32", F32_TOL), ("split", SPLIT_TOL)):
        m, _ = make(cfg, weights=w, precision=precision, max_tokens=64 * 44, max_batch=22)
        seqs = [0] + [m.seq_create() for _ in range(21)]
        for s, p in zip(seqs, prompts):
            m.step_batch([(s, p[:-4], [])])
        for t in range(4, 0, -1):
            live = range(22) if t > 2 else range(3, 12)
            lg = m.step_batch([(seqs[i], [prompts[i][-t]], [0]) for i in live])
            for r, i in enumerate(live):
                assert rel(lg[r], want[i][len(prompts[i]) - t]) < tol, (t, i)
        m.close()


@pytest.mark.gpu
def test_pages_and_slots_are_used_again():
    m, w = make(FULL, 13, precision="f32", max_tokens=256, max_batch=2)        # 4 pages, 2 slots
    a, b, c = (tokens(n, FULL["vocab"], 30 + i) for i, n in enumerate((130, 120, 100)))
    s1 = m.seq_create()
    m.step_batch([(0, a, []), (s1, b[:60], [])])                # 3 + 1 pages: the pool is full
    with pytest.raises(Exception):
        m.step_batch([(s1, b[60:], [])])                        # needs a fifth page: refused, nothing changes
    assert m.seq_len(s1) == 60
    m.clear_kv_cache()                                          # sequence 0 gives its three pages back
    got_b = m.step_batch([(s1, b[60:], [len(b) - 61])])
    assert rel(got_b[0], oracle_logits(FULL, w, b)[-1]) < F32_TOL
    m.seq_free(s1)
    s2 = m.seq_create()                                         # same slot: input rings and states start from zero, pages still hold b's rows
    assert s2 == s1
    got_c = m.step_batch([(s2, c[:50], []), (0, a[:64], [63])])
    got_c2 = m.step_batch([(s2, c[50:], [49])])
    assert rel(got_c2[0], oracle_logits(FULL, w, c)[-1]) < F32_TOL
    assert rel(got_c[0], oracle_logits(FULL, w, a[:64])[-1]) < F32_TOL
    m.close()


@pytest.mark.gpu
def test_scratch_pages_of_built_keys_are_used_again():
    # serving precision: built keys and values live on scratch pages shared by layers of unequal widths; pages change hands between requests
    cfg = config([layer(latent(heads=4, dim=24, rot_dim=8, vdim=40, kv_rank=32, size=40, scale=0.6)), layer(latent(heads=2, dim=48, rot_dim=16, vdim=16, kv_rank=40, size=90, scale=0.4))], streams=2)
    m, w = make(cfg, 14, precision="split", max_tokens=320, max_batch=2)
    s1 = m.seq_create()
    for k in range(3):
        a, b = tokens(150, cfg["vocab"], 80 + k), tokens(110, cfg["vocab"], 90 + k)
        wa, wb = oracle_logits(cfg, w, a), oracle_logits(cfg, w, b)
        g = m.step_batch([(0, a[:70], all_rows(70)), (s1, b[:40], all_rows(40))])
        h = m.step_batch([(s1, b[40:], all_rows(70)), (0, a[70:], all_rows(80))])
        assert rel(np.concatenate([g[:70], h[70:]]), wa) < SPLIT_TOL and rel(np.concatenate([g[70:], h[:70]]), wb) < SPLIT_TOL, k
        m.clear_kv_cache()
        m.seq_free(s1)
        s1 = m.seq_create()
    m.close()


@pytest.mark.gpu
def test_window_edges_page_borders_and_carried_states_with_sharp_scores():
    cfg, w = sharp_model(41)                                    # windows of 33, 41 and 64 keys
    m, _ = make(cfg, weights=w, max_tokens=1024, max_batch=2, precision="f32")
    ids = tokens(330, cfg["vocab"], 42)
    want = oracle_logits(cfg, w, ids)
    got = m.step_batch([(0, ids, all_rows(330))])
    assert rel(got, want) < F32_TOL
    # decode over the borders of 32-key tiles and 64-token pages and the places where a window's far edge crosses them, after a prompt
    # that ends just before / on / after them
    for start in (1, 2, 3, 31, 32, 33, 34, 40, 41, 42, 63, 64, 65, 66, 72, 73, 95, 96, 97, 104, 105, 127, 128, 129, 191, 192, 193, 255, 256, 257):
        m.clear_kv_cache()
        m.step_batch([(0, ids[:start], [])])
        rows = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[start:start + 4]])
        assert rel(rows, want[start:start + 4]) < F32_TOL, start
    # the same edges inside portions of a prompt, the second portion as short as two tokens
    for cut in (33, 34, 41, 64, 65, 97, 129, 256):
        m.clear_kv_cache()
        a = m.step_batch([(0, ids[:cut - 1], [cut - 2])])
        b = m.step_batch([(0, ids[cut - 1:cut + 1], all_rows(2))])
        c = m.step_batch([(0, ids[cut + 1:cut + 40], all_rows(39))])
        assert rel(np.concatenate([a, b, c]), want[cut - 2:cut + 40]) < F32_TOL, cut
    m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("shape", TENSOR_CORE_SHAPES)
def test_sharp_scores_through_the_tensor_core_attention(shape):
    cfg, w, ids = sharp_attention(*shape)
    want = oracle_logits(cfg, w, ids)
    m, _ = make(cfg, weights=w, precision="split")
    assert rel(m.step_batch([(0, ids, all_rows(260))]), want) < SPLIT_TOL
    m.clear_kv_cache()
    a = m.step_batch([(0, ids[:131], all_rows(131))])
    b = m.step_batch([(0, ids[131:199], all_rows(68))])
    c = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[199:]])
    assert rel(np.concatenate([a, b, c]), want) < SPLIT_TOL
    m.close()


@pytest.mark.gpu
def test_keys_far_away_without_a_window():
    cfg, w = sharp_model(43, far=True)
    ids = tokens(900, cfg["vocab"], 44)
    want = oracle_logits(cfg, w, ids)
    # (scores this sharp multiply rounding: one f32 rounding of the scores or of the carried state alone moves these logits by 6e-6)
    for precision, tol in (("f32", 1e-4), ("split", SPLIT_TOL)):
        m, _ = make(cfg, weights=w, max_tokens=2048, precision=precision)
        got = m.step_batch([(0, ids[:700], [300, 500, 699])])
        assert rel(got, want[[300, 500, 699]]) < tol
        rows = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[700:800]])      # 100 decoded tokens, the context split over blocks
        assert rel(rows, want[700:800]) < tol
        got = m.step_batch([(0, ids[800:], all_rows(100))])                                # a portion that builds keys for 800 tokens before it
        assert rel(got, want[800:]) < tol
        m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("precision,tol", [("f32", F32_TOL), ("split", SPLIT_TOL)])
def test_long_portions_on_carried_states(precision, tol):
    # more than a thousand rows in a step, on states that an earlier portion left, beside a short request, with lengths that leave the
    # last tile of rows ragged
    cfg = config([layer(parallel(heads=2, kv_heads=1, dim=16, vdim=16, right=recurrence(200, 1, 3)), None),
                  layer(latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=20, size=50), 40)], width=96, vocab=150)
    w = O.random_weights(cfg, 27)
    w["l0.mix.right.lam"] = bf(w["l0.mix.right.lam"] - 2.0)
    m, _ = make(cfg, weights=w, precision=precision, max_tokens=2048)
    ids, other = tokens(1400, cfg["vocab"], 28), tokens(40, cfg["vocab"], 29)
    want, want2 = oracle_logits(cfg, w, ids), oracle_logits(cfg, w, other)
    s1 = m.seq_create()
    a = m.step_batch([(0, ids[:100], [99])])
    b = m.step_batch([(s1, other[:30], [29]), (0, ids[100:1203], [0, 350, 1102])])
    c = m.step_batch([(0, ids[1203:1399], [0, 195]), (s1, other[30:], [9])])
    d = m.step_batch([(0, ids[1399:], [0])])
    assert rel(np.concatenate([a, b[1:], c[:2], d]), want[[99, 100, 450, 1202, 1203, 1398, 1399]]) < tol
    assert rel(np.stack([b[0], c[2]]), want2[[29, 39]]) < tol
    m.close()


@pytest.mark.gpu
def test_strong_and_weak_decays():
    # decays from one (nothing forgotten, nothing taken in) to zero (everything forgotten) side by side
    cfg = config([layer(parallel(right=recurrence(48, 2, 4)), None), layer(parallel(right=recurrence(30, 1, 2)), None)])
    w = O.random_weights(cfg, 33)
    for li in (0, 1):
        w[f"l{li}.mix.right.lam"][::3] = 20.0
        w[f"l{li}.mix.right.lam"][1::3] = -20.0
    ids = tokens(300, cfg["vocab"], 34)
    want = oracle_logits(cfg, w, ids)
    assert np.isfinite(want).all()
    for precision, tol in (("f32", F32_TOL), ("split", SPLIT_TOL)):
        m, _ = make(cfg, weights=w, precision=precision)
        assert rel(m.step_batch([(0, ids, all_rows(300))]), want) < tol
        m.clear_kv_cache()
        a = m.step_batch([(0, ids[:290], all_rows(290))])
        b = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[290:]])
        assert rel(np.concatenate([a, b]), want) < tol
        m.close()


@pytest.mark.gpu
def test_first_tokens_of_a_sequence():
    m, w = make(FULL, 15, precision="f32")
    ids = tokens(7, FULL["vocab"], 16)
    want = oracle_logits(FULL, w, ids)
    assert rel(m.step_batch([(0, ids[:1], [0])]), want[:1]) < F32_TOL           # a one-token prompt: zeros before the convolution, an empty memory
    assert rel(m.step_batch([(0, ids[1:2], [0])]), want[1:2]) < F32_TOL
    assert rel(m.step_batch([(0, ids[2:4], [0, 1])]), want[2:4]) < F32_TOL      # a portion shorter than the convolution
    assert rel(m.step_batch([(0, ids[4:], [0, 1, 2])]), want[4:]) < F32_TOL
    m.close()


@pytest.mark.gpu
def test_greedy_generation_through_generate_and_the_scheduler():
    from crane_b200.scheduler import BatchScheduler
    m, w = make(FULL, 19, precision="f32", max_tokens=512)

    def oracle_greedy(prompt, n):
        s = O.State(FULL)
        lg = oracle_logits(FULL, w, prompt, s)[-1]
        out, margins = [], []
        for _ in range(n):
            top = np.sort(lg)[-2:]
            margins.append(top[1] - top[0])
            out.append(int(lg.argmax()))
            lg = oracle_logits(FULL, w, [out[-1]], s)[-1]
        return out, min(margins)

    prompts = [tokens(n, FULL["vocab"], 50 + i) for i, n in enumerate((70, 9, 33, 130, 20, 64))]
    want = [oracle_greedy(p, 12) for p in prompts]
    assert min(mg for _, mg in want) > 1e-4                     # no decision of this test is a close call
    assert m.generate(prompts[0], max_new_tokens=12).tolist() == want[0][0]
    m.clear_kv_cache()
    sch = BatchScheduler(m, chunk=48, max_live=3, token_budget=80)
    rids = [sch.add(p, 12) for p in prompts]
    out = sch.run()
    for rid, (toks, _) in zip(rids, want):
        assert out[rid] == toks, rid
    sch = BatchScheduler(m, chunk=32, max_live=2)
    rid = sch.add(prompts[1], 6, temperature=0.8, top_k=1, seed=3)         # top-k 1 is greedy whatever the draw
    assert sch.run()[rid] == want[1][0][:6]
    m.clear_kv_cache()
    s1 = m.seq_create()
    m.step_batch([(0, prompts[2], []), (s1, prompts[4], [])])
    first = [want[2][0][0], want[4][0][0]]
    toks, _ = m.decode_batch([0, s1], first, n_steps=5)                     # the graph-replayed loop, two sequences side by side
    assert toks[0].tolist() == want[2][0][1:6] and toks[1].tolist() == want[4][0][1:6]
    m.close()


@pytest.mark.gpu
def test_wide_layers_take_the_tensor_core_paths():
    # widths of a real model's layers in small numbers
    cfg = config([layer(latent(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=256, size=150, scale=0.07), 352),
                  layer(parallel(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.12, right=recurrence(256, 2, 4)), 64),
                  layer(latent(heads=2, dim=64, rot_dim=32, vdim=64, kv_rank=512, size=100, scale=0.1), 128),
                  layer(parallel(heads=4, kv_heads=1, dim=128, vdim=256, scale=0.09, right=recurrence(320, 1, 4)), None)], width=256, vocab=300, loop=(1, 3, 2))
    m, w = make(cfg, 21, precision="split")
    ids = tokens(400, cfg["vocab"], 22)
    want = oracle_logits(cfg, w, ids)
    assert rel(m.step_batch([(0, ids, all_rows(400))]), want) < SPLIT_TOL
    m.clear_kv_cache()
    a = m.step_batch([(0, ids[:333], all_rows(333))])
    b = m.step_batch([(0, ids[333:390], all_rows(57))])
    c = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[390:]])
    assert rel(np.concatenate([a, b, c]), want) < SPLIT_TOL
    m.close()


def random_config(seed):
    """A layer list drawn at random: the two mixers in any order, widths that are and are not multiples of 4 and 8, every grouping of
    heads, windows around tile and page sizes, with and without a feed-forward, any span repeated."""
    r = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(r.integers(len(xs)))]
    layers = []
    for _ in range(int(r.integers(1, 6))):
        if pick(0, 1):
            dr = pick(2, 6, 8, 16, 32)
            layers.append(layer(latent(heads=pick(1, 2, 3, 5, 8), dim=pick(7, 16, 24, 40, 64), rot_dim=dr, vdim=pick(6, 15, 24, 64, 80), kv_rank=pick(5, 16, 33, 64, 96),
                                       size=pick(0, 1, 5, 31, 32, 33, 64, 100), scale=float(pick(0.1, 0.3, 0.6)), base=float(pick(100.0, 1e4, 1e6))), pick(0, 12, 30, 64)))
        else:
            G, d = pick(1, 2, 3), pick(8, 18, 32, 40, 64)
            k = pick(1, 2, 4)
            layers.append(layer(parallel(heads=G * pick(1, 2, 4), kv_heads=G, dim=d, vdim=pick(8, 20, 33, 64, 128), scale=float(pick(0.1, 0.3, 0.6)), base=float(pick(100.0, 1e4, 1e6)),
                                         dims=min(d, pick(2, 8, 16, 64)), left_scale=float(pick(0.3, 1.0)), right_scale=float(pick(0.5, 1.0, 1.5)),
                                         right=recurrence(k * pick(5, 16, 33, 72, 140), k, pick(1, 2, 3, 4, 5))), pick(0, 12, 30, 64)))
    n = len(layers)
    a = int(r.integers(0, n))
    return config(layers, width=pick(72, 96, 120, 160), vocab=pick(90, 211, 300), eps=float(pick(1e-6, 1e-5)), streams=pick(1, 2, 3, 4), logit_scale=float(pick(0.2, 1.0)),
                  loop=pick(None, (a, int(r.integers(a, n)) + 1, pick(1, 2, 3))))


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(10))
def test_random_layer_lists(seed):
    cfg = random_config(100 + seed)
    r = np.random.default_rng(seed)
    ids, other = tokens(150, cfg["vocab"], 200 + seed), tokens(70, cfg["vocab"], 300 + seed)
    w = O.random_weights(cfg, 400 + seed)
    want, want2 = oracle_logits(cfg, w, ids), oracle_logits(cfg, w, other)
    for precision, tol in (("f32", F32_TOL), ("split", SPLIT_TOL)):
        m, _ = make(cfg, weights=w, precision=precision)
        assert rel(m.step_batch([(0, ids, all_rows(150))]), want) < tol, (precision, "whole")
        m.clear_kv_cache()
        s1 = m.seq_create()
        at, at2, rows, rows2 = 0, 0, [], []
        while at < 150:                                      # random cuts, the second request beside some of them
            c = int(min(150 - at, r.choice([1, 2, 3, 17, 40, 64])))
            entries = [(0, ids[at:at + c], all_rows(c))]
            c2 = int(min(70 - at2, r.choice([0, 1, 2, 30])))
            if c2:
                entries.append((s1, other[at2:at2 + c2], all_rows(c2)))
            lg = m.step_batch(entries)
            rows.append(lg[:c]); rows2.append(lg[c:]); at += c; at2 += c2
        assert rel(np.concatenate(rows), want) < tol, (precision, "cuts")
        got2 = np.concatenate(rows2)
        assert rel(got2, want2[:len(got2)]) < tol, (precision, "beside")
        m.close()


@pytest.mark.gpu
def test_configurations_and_tensors_that_do_not_fit_are_refused():
    import crane_b200

    def refused(change):
        cfg = config([layer(latent()), layer(parallel())])
        change(cfg)
        with pytest.raises(crane_b200.CraneB200Error):
            crane_b200.RupulixModel(cfg, device=0, max_tokens=256).close()
    refused(lambda c: c["layers"][0].update(type="other"))
    refused(lambda c: c["layers"][1]["mixer"]["left"].update(heads=3, kv_heads=2))
    refused(lambda c: c["layers"][1]["mixer"].pop("right"))
    refused(lambda c: c["layers"][1]["mixer"]["right"].update(blocks=7))
    refused(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8))
    refused(lambda c: c["layers"][0]["mixer"].update(kv_rank=0))
    refused(lambda c: c["layers"][0]["mixer"]["mask"].update(size=-1))
    refused(lambda c: c["layers"][1]["mlp"].update(kind="moe"))
    refused(lambda c: c.update(streams=0))
    refused(lambda c: c.update(loop={"start": 1, "stop": 3, "times": 2}))
    cfg = config([layer(latent()), layer(parallel())])
    w = O.random_weights(cfg, 1)
    m = crane_b200.RupulixModel(cfg, device=0, max_tokens=256)
    t = lambda k: w[k].to(torch.float32).numpy()
    m.load_tensor("l1.mix.right.ra", t("l1.mix.right.ra"))
    with pytest.raises(crane_b200.CraneB200Error):
        m.load_tensor("l1.mix.right.ri", np.zeros((3, 20, 19), np.float32))
    with pytest.raises(crane_b200.CraneB200Error):
        m.load_tensor("l0.hc1.mix", np.zeros((3, 2), np.float32))
    with pytest.raises(crane_b200.CraneB200Error):
        m.load_tensor("l0.mix.extra", t("l0.mix.sink"))
    with pytest.raises(crane_b200.CraneB200Error):
        m.finalize()
    m.close()


@pytest.mark.gpu
def test_model_folder_loader_and_trace_runner(tmp_path):
    import json, os, subprocess, sys
    cfg, w = FULL, O.random_weights(FULL, 23)
    hdr, blob = {}, b""
    for k, t in w.items():
        bits = O.to_numpy_bf16_bits(t).tobytes()
        hdr[k] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [len(blob), len(blob) + len(bits)]}
        blob += bits
    mdir = tmp_path / "model"; mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(cfg))
    h = json.dumps(hdr).encode()
    (mdir / "model.safetensors").write_bytes(len(h).to_bytes(8, "little") + h + blob)
    a, b = tokens(80, cfg["vocab"], 24), tokens(70, cfg["vocab"], 25)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [49]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [0, 67]}, {"id": "a", "tokens": a[50:51], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[51:], "want": []}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [69]}], "end": ["c"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(mdir), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    wa, wb = oracle_logits(cfg, w, a), oracle_logits(cfg, w, b)
    read = lambda n: np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    assert rel(read(0), wa[49:50]) < F32_TOL
    assert rel(read(1), np.stack([wb[2], wb[69], wa[50]])) < F32_TOL
    assert not (out / "2.f32").exists()
    assert rel(read(3), wb[69:70]) < F32_TOL                    # request c runs on the slot and pages b gave back
