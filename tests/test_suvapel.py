"""Suvapel (Dynamic-Tanh layers whose mixer and feed-forward join the stream together; the gated delta rule, windowed attention with
kept first tokens beside a delta rule with a decay per key channel; a token embedding behind every layer) against the plain oracle of
oracle/suvapel.py.

Small configurations with their own random weights; the oracle runs in float64.  The engine's "f32" precision is held to a tight
bar (a window one token off, a lost first token, a state of the wrong slot, a bias on the wrong row shows), the serving precision to
the bar its operand rounding allows.
"""
import copy
import math

import numpy as np
import pytest
import torch

from oracle import suvapel as O

T64 = torch.float64


# ---------------------------------------------------------------------------------------------------- configurations
def rule(heads=3, kv_heads=1, dim=20, vdim=28, conv=4, **kw):
    return dict({"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, **kw)


def yarn(dims=16, base=10000.0, scaling=True, factor=4.0, original=96, fast=8.0, slow=1.0):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return r


def delta(**kw):
    return {"type": "delta", "mixer": rule(**kw)}


def parallel(heads=6, kv_heads=2, dim=24, vdim=40, conv=3, size=37, keep=5, rot=None, scale=0.2, left_scale=0.7, right_scale=1.2, right=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rot": rot or yarn(), "scale": scale}
    if size:
        left["mask"] = {"size": size, "keep_first": keep}
    return {"type": "parallel", "mixer": {"left": left, "right": right or rule(heads=4, kv_heads=2, dim=12, vdim=20), "left_scale": left_scale, "right_scale": right_scale}}


def layer(mx, ff=52):
    return dict(copy.deepcopy(mx), mlp={"kind": "dense", "ff": ff} if ff else None)


def config(layers, width=120, vocab=211, eps=1e-5, mult=0.6, side=10):
    return {"architecture": "Suvapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "token_side": {"dim": side},
            "layers": copy.deepcopy(layers)}


# five layers of unequal geometry, every mixer at least twice, one layer without a feed-forward
FULL = config([layer(delta()),
               layer(parallel()),
               layer(parallel(heads=2, kv_heads=2, dim=16, vdim=8, conv=4, size=70, keep=1, rot=yarn(dims=8, base=500.0, factor=2.0, original=40, fast=4.0), scale=0.3,
                              right=rule(heads=2, kv_heads=2, dim=9, vdim=7, conv=2, a_rank=5, g_rank=17)), None),
               layer(delta(heads=4, kv_heads=4, dim=7, vdim=12, conv=3), 30),
               layer(parallel(heads=3, kv_heads=1, dim=18, vdim=21, conv=2, size=33, keep=33, rot=yarn(dims=18), right=rule(heads=3, kv_heads=1, dim=33, vdim=18, conv=3)), 64)])
SINGLE = {
    "delta_only": config([layer(delta(), None)]),
    "delta_every_head_its_own_keys_one_tap": config([layer(delta(heads=2, kv_heads=2, dim=16, vdim=16, conv=1), None)], width=72, vocab=90),
    "delta_five_taps_one_channel": config([layer(delta(heads=1, kv_heads=1, dim=1, vdim=3, conv=5))], width=32, vocab=50, side=3),
    "delta_wide": config([layer(delta(heads=2, kv_heads=1, dim=130, vdim=150, conv=4), None)], width=64, vocab=128),
    "delta_widest_keys": config([layer(delta(heads=1, kv_heads=1, dim=256, vdim=20, conv=2), None)], width=64, vocab=70),
    "parallel_only": config([layer(parallel(), None)]),
    "parallel_window_one_keeps_two": config([layer(parallel(heads=1, kv_heads=1, dim=16, vdim=16, size=1, keep=2), 24)], width=64, vocab=70),
    "parallel_keeps_none": config([layer(parallel(size=20, keep=0))]),
    "parallel_no_window": config([layer(parallel(heads=4, kv_heads=1, dim=13, vdim=21, size=0, rot=yarn(dims=6)), None)], width=66, vocab=90),
    "parallel_keeps_more_than_the_window": config([layer(parallel(size=7, keep=45), None)]),
    "parallel_one_tap_plain_rotation": config([layer(parallel(conv=1, rot=yarn(dims=24, scaling=False), right=rule(heads=1, kv_heads=1, dim=8, vdim=64, conv=1, a_rank=1, g_rank=2)))]),
    "parallel_long_convolutions": config([layer(parallel(conv=6, right=rule(heads=2, kv_heads=1, dim=40, vdim=5, conv=7, a_rank=30, g_rank=3)), None)]),
    "parallel_window_longer_than_the_prompt": config([layer(parallel(size=500, keep=3))]),
    "side_of_one_column": config([layer(delta(), 200)], width=96, vocab=100, side=1, mult=1.0),
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


def sharp_model(seed, size=33, keep=4, far=False):
    """Scores with a spread of several units (a query looks at one or two keys of what it sees, wherever they are), slow decays (the
    delta rules remember hundreds of tokens): a key just inside or just outside a window, a kept first token, a state that was not
    carried moves the logits by O(1).  far: no window, single keys hundreds of tokens back carry the output."""
    cfg = config([layer(parallel(heads=4, kv_heads=2, dim=24, vdim=24, size=0 if far else size, keep=keep, scale=1.6, rot=yarn(dims=8, base=1e5, original=200)), None),
                  layer(delta(heads=2, kv_heads=1, dim=16, vdim=24), 40),
                  layer(parallel(heads=4, kv_heads=1, dim=16, vdim=32, size=0 if far else size + 8, keep=keep + 31, scale=1.9, rot=yarn(dims=4, base=1e6, scaling=False)), None),
                  layer(parallel(heads=2, kv_heads=1, dim=32, vdim=16, size=0 if far else 64, keep=1, scale=1.4, rot=yarn(dims=8, base=1e5, original=100)))], width=128, vocab=200)
    w = O.random_weights(cfg, seed)
    for k in w:
        if k.endswith("A_log"):
            w[k] = bf(w[k] - 3.0)
        if k.endswith("left.q") or k.endswith("left.k"):
            w[k] = bf(w[k] * 1.5)
        if k.endswith("left.o"):
            w[k] = bf(w[k] * 2.0)
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
    # the norm squashes every entry on its own
    y = O.dyt(torch.tensor([0.0, 100.0, -100.0], dtype=T64), torch.tensor(2.0, dtype=T64), torch.tensor([3., 4., 5.], dtype=T64), torch.tensor([0.5, 0., 1.], dtype=T64))
    assert torch.allclose(y, torch.tensor([0.5, 4.0, -4.0], dtype=T64))
    # causal convolution: the last column weighs the current token, the window carries the inputs before the portion
    u = torch.tensor([[1.], [2.], [4.]], dtype=T64)
    cv, win = O.causal_conv(u, torch.tensor([[100., 10., 1.]], dtype=T64), torch.tensor([[7.], [8.]], dtype=T64))
    assert cv[:, 0].tolist() == [781., 812., 124.] and win[:, 0].tolist() == [2., 4.]
    # rotation: dimension i turns with dimension i + dims / 2, the rest passes
    x = torch.tensor([[[1., 2., 0., 0., 9.]]], dtype=T64)
    y = O.rotate(x, torch.tensor([3]), {"dims": 4, "base": 100.0})
    assert torch.allclose(y[0, 0], torch.tensor([math.cos(3.), 2 * math.cos(.3), math.sin(3.), 2 * math.sin(.3), 9.], dtype=T64))
    # scaled frequencies: pairs that turn often keep theirs, pairs that hardly turn are slowed by the factor, a ramp between
    f, mag = O.rotation({"dims": 8, "base": 10.0 ** 4, "scaling": {"factor": 4.0, "original": 2 * math.pi * 100, "fast": 10.0, "slow": 0.1}})
    assert np.allclose(f, [1.0, 0.1 * (1 / 4) * 0 + 0.1, 0.01 * (0.5 / 4 + 0.5), 0.001 / 4]) and abs(mag - (0.1 * math.log(4) + 1)) < 1e-12
    f, mag = O.rotation({"dims": 4, "base": 100.0})
    assert np.allclose(f, [1.0, 0.1]) and mag == 1.0
    # visibility: the window holds `size` keys with the row's own, the first tokens stay
    assert O.visible(9, {"size": 3, "keep_first": 2}).tolist() == [0, 1, 7, 8, 9]
    assert O.visible(3, {"size": 3, "keep_first": 2}).tolist() == [0, 1, 2, 3]
    assert O.visible(4, {"size": 1}).tolist() == [4] and O.visible(2, None).tolist() == [0, 1, 2]
    # softmax attention with two visible keys of equal scores
    q = torch.ones(1, 1, 2, dtype=T64)
    k = torch.tensor([[[1., 0.]], [[5., 5.]], [[0., 1.]]], dtype=T64)
    v = torch.tensor([[[2., 0.]], [[100., 0.]], [[0., 6.]]], dtype=T64)
    assert torch.allclose(O.attend(q, k, v, [2], 1.0, {"size": 1, "keep_first": 1})[0, 0], torch.tensor([1., 3.], dtype=T64))
    # delta rule by hand: writing v under a unit key stores it; writing again under the same key replaces what the decay left of it
    one = torch.ones(2, dtype=T64)
    kk = torch.tensor([[1., 0.], [1., 0.]], dtype=T64)
    o, S = O.delta_rule(2 * kk, kk, torch.tensor([[4.], [10.]], dtype=T64), one, torch.tensor([[1., 1.], [.5, 1.]], dtype=T64), torch.zeros(2, 1, dtype=T64))
    assert o[:, 0].tolist() == [8.0, 20.0] and S[:, 0].tolist() == [10.0, 0.0]
    o, S = O.delta_rule(kk[:1], kk[:1], torch.tensor([[4.]], dtype=T64), 0.5 * one[:1], torch.tensor([[.5, .25]], dtype=T64), torch.tensor([[2.], [8.]], dtype=T64))
    assert S[:, 0].tolist() == [1.0 + 0.5 * (4.0 - 1.0), 2.0] and o[0, 0] == 2.5
    # unit vectors (their constant shows on small ones), root mean square, the activations
    assert torch.allclose(O.unit(torch.tensor([3., 4.], dtype=T64) * 1e-3), torch.tensor([3., 4.], dtype=T64) * 1e-3 / math.sqrt(25e-6 + 1e-6))
    assert torch.allclose(O.rms(torch.tensor([3., 4.], dtype=T64), 0.5), torch.tensor([3., 4.], dtype=T64) / math.sqrt(13.0))
    z = torch.tensor([1.3, -0.7], dtype=T64)
    assert torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh")) and torch.allclose(O.silu(z), torch.nn.functional.silu(z))
    # the feed-forward's three biases
    p = {"gate": torch.eye(2, dtype=T64), "gate.b": one, "up": 2 * torch.eye(2, dtype=T64), "up.b": -one, "down": torch.eye(2, dtype=T64), "down.b": 3 * one}
    assert torch.allclose(O.feed_forward(z[None], p, ""), O.silu(z + 1) * (2 * z - 1) + 3)


def test_oracle_sees_what_the_sharp_tests_are_about():
    cfg, w = sharp_model(41)
    ids = tokens(200, cfg["vocab"], 42)
    base = oracle_logits(cfg, w, ids)
    for li, what, by in ((0, "size", 1), (0, "size", -1), (2, "size", 1), (3, "size", -1), (0, "keep_first", 1), (0, "keep_first", -1), (2, "keep_first", -1), (3, "keep_first", -1)):
        other = copy.deepcopy(cfg)
        other["layers"][li]["mixer"]["left"]["mask"][what] += by
        assert rel(oracle_logits(other, w, ids)[80:], base[80:]) > 5e-3, (li, what, by)
    for li in (0, 1, 2):                                             # delta states that were not carried over a cut, a lost window of a convolution
        lost = O.State(cfg)
        oracle_logits(cfg, w, ids[:120], lost)
        lost.mem[li] = [torch.zeros_like(S) for S in lost.mem[li]]
        assert rel(oracle_logits(cfg, w, ids[120:], lost), base[120:]) > 1e-2
        lost = O.State(cfg)
        oracle_logits(cfg, w, ids[:120], lost)
        lost.win[li] = {k: torch.zeros_like(v) for k, v in lost.win[li].items()}
        assert rel(oracle_logits(cfg, w, ids[120:], lost), base[120:]) > 1e-2
    cfg, w = sharp_model(43, far=True)                                # no window: single keys hundreds of tokens back carry the output
    ids = tokens(400, cfg["vocab"], 44)
    base = oracle_logits(cfg, w, ids)
    near = copy.deepcopy(cfg)
    near["layers"][0]["mixer"]["left"]["mask"] = {"size": 200, "keep_first": 0}
    assert rel(oracle_logits(near, w, ids)[300:], base[300:]) > 1e-2


TENSOR_CORE_SHAPES = [(64, 64, 40, 3), (64, 128, 100, 40), (128, 64, 65, 64), (128, 128, 33, 70), (64, 128, 31, 1)]      # dim, vdim, window, kept tokens


def sharp_attention(dim, vdim, size, keep):
    cfg = config([layer(parallel(heads=4, kv_heads=2, dim=dim, vdim=vdim, size=size, keep=keep, scale=5.0 / math.sqrt(dim), rot=yarn(dims=dim // 4, base=1e6)), None)], width=128, vocab=150)
    w = O.random_weights(cfg, 45)
    for k, by in (("q", 1.5), ("k", 1.5), ("o", 4.0)):
        w[f"l0.mix.left.{k}"] = bf(w[f"l0.mix.left.{k}"] * by)
    return cfg, w, tokens(260, cfg["vocab"], 46)


@pytest.mark.parametrize("shape", TENSOR_CORE_SHAPES)
def test_oracle_sees_the_edges_of_the_tensor_core_tests(shape):
    cfg, w, ids = sharp_attention(*shape)
    want = oracle_logits(cfg, w, ids)
    for what, by in (("size", 1), ("size", -1), ("keep_first", -1), ("keep_first", 1)):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["left"]["mask"][what] += by
        assert rel(oracle_logits(other, w, ids)[150:], want[150:]) > 10 * SPLIT_TOL, (what, by)


# ---------------------------------------------------------------------------------------------------- GPU
def make(cfg, seed=0, weights=None, **opts):
    import crane_b200
    w = weights or O.random_weights(cfg, seed)
    opts.setdefault("max_tokens", 1024)
    opts.setdefault("max_batch", 4)
    m = crane_b200.SuvapelModel(cfg, device=0, **opts)
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
    m, w = make(FULL, 9, precision="f32")
    n = sum(cuts)
    ids = tokens(n, FULL["vocab"], 10)
    want = oracle_logits(FULL, w, ids)
    at, rows = 0, []
    for c in cuts:
        rows.append(m.step_batch([(0, ids[at:at + c], all_rows(c))]))
        at += c
    assert rel(np.concatenate(rows), want) < F32_TOL
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
    s2 = m.seq_create()                                         # same slot: windows and states start from zero, pages still hold b's rows
    assert s2 == s1
    got_c = m.step_batch([(s2, c[:50], []), (0, a[:64], [63])])
    got_c2 = m.step_batch([(s2, c[50:], [49])])
    assert rel(got_c2[0], oracle_logits(FULL, w, c)[-1]) < F32_TOL
    assert rel(got_c[0], oracle_logits(FULL, w, a[:64])[-1]) < F32_TOL
    m.close()


@pytest.mark.gpu
def test_window_edges_kept_tokens_page_borders_and_carried_states_with_sharp_scores():
    cfg, w = sharp_model(41)                                    # windows of 33, 41 and 64 keys; 4, 35 and 1 first tokens kept
    m, _ = make(cfg, weights=w, max_tokens=1024, max_batch=2, precision="f32")
    ids = tokens(330, cfg["vocab"], 42)
    want = oracle_logits(cfg, w, ids)
    got = m.step_batch([(0, ids, all_rows(330))])
    assert rel(got, want) < F32_TOL
    # decode over the borders of 32-key tiles and 64-token pages and the places where a window's far edge crosses them or leaves the
    # kept tokens, after a prompt that ends just before / on / after them
    for start in (1, 2, 3, 4, 5, 31, 32, 33, 34, 35, 36, 37, 38, 40, 41, 42, 63, 64, 65, 66, 68, 72, 75, 76, 77, 95, 96, 97, 104, 105, 127, 128, 129, 191, 192, 193, 255, 256, 257):
        m.clear_kv_cache()
        m.step_batch([(0, ids[:start], [])])
        rows = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[start:start + 4]])
        assert rel(rows, want[start:start + 4]) < F32_TOL, start
    # the same edges inside portions of a prompt, the second portion as short as two tokens
    for cut in (33, 34, 37, 41, 64, 65, 76, 97, 129, 256):
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
    m, _ = make(cfg, weights=w, max_tokens=2048, precision="f32")
    ids = tokens(900, cfg["vocab"], 44)
    want = oracle_logits(cfg, w, ids)
    got = m.step_batch([(0, ids[:700], [300, 500, 699])])
    assert rel(got, want[[300, 500, 699]]) < F32_TOL
    rows = np.concatenate([m.step_batch([(0, [t], [0])]) for t in ids[700:]])          # 200 decoded tokens, the context split over blocks
    assert rel(rows, want[700:]) < F32_TOL
    m.close()


@pytest.mark.gpu
@pytest.mark.parametrize("precision,tol", [("f32", F32_TOL), ("split", SPLIT_TOL)])
def test_long_portions_on_carried_states(precision, tol):
    # more than a thousand rows in a step, on states that an earlier portion left, beside a short request, with lengths that leave the
    # last tile of rows ragged
    cfg = config([layer(delta(heads=2, kv_heads=1, dim=18, vdim=21, conv=3), None),
                  layer(parallel(heads=2, kv_heads=1, dim=16, vdim=16, size=50, keep=9, right=rule(heads=2, kv_heads=2, dim=32, vdim=32)), 40)], width=96, vocab=150)
    w = O.random_weights(cfg, 27)
    for k in w:
        if k.endswith("A_log"):
            w[k] = bf(w[k] - 2.0)
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
    # decays from one (nothing forgotten) to zero (everything forgotten), also side by side on the key channels of one head
    cfg = config([layer(parallel(right=rule(heads=2, kv_heads=1, dim=24, vdim=16)), None), layer(delta(heads=3, kv_heads=3, dim=12, vdim=12), None)])
    w = O.random_weights(cfg, 33)
    d = w["l0.mix.right.dt_bias"]
    d[::3] = 30.0
    d[1::3] = -30.0
    w["l1.mix.dt_bias"] = bf(torch.tensor([40.0, -30.0, 0.0], dtype=T64))
    w["l1.mix.A_log"] = bf(torch.tensor([3.0, -5.0, 1.0], dtype=T64))
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
    assert rel(m.step_batch([(0, ids[:1], [0])]), want[:1]) < F32_TOL           # a one-token prompt: zeros in every window, an empty memory
    assert rel(m.step_batch([(0, ids[1:2], [0])]), want[1:2]) < F32_TOL
    assert rel(m.step_batch([(0, ids[2:4], [0, 1])]), want[2:4]) < F32_TOL      # a portion shorter than the convolution's window
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
    # widths the tensor-core kernels take: 64- and 128-wide heads, many rows; wide delta states, low ranks of a real model's size
    cfg = config([layer(parallel(heads=4, kv_heads=2, dim=64, vdim=64, size=100, keep=10, scale=0.12, right=rule(heads=2, kv_heads=2, dim=128, vdim=128, a_rank=128, g_rank=64)), 352),
                  layer(delta(heads=4, kv_heads=2, dim=64, vdim=96, conv=4), 64),
                  layer(parallel(heads=2, kv_heads=1, dim=128, vdim=128, size=150, keep=2, scale=0.09, right=rule(heads=2, kv_heads=1, dim=64, vdim=64, conv=3, a_rank=300, g_rank=260)), 128),
                  layer(parallel(heads=4, kv_heads=4, dim=64, vdim=128, size=0, scale=0.1), None)], width=256, vocab=300, side=40)
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
    heads, windows and kept tokens around tile and page sizes, with and without a feed-forward."""
    r = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(r.integers(len(xs)))]

    def some_rule(**kw):
        G = pick(1, 2, 3)
        return rule(heads=G * pick(1, 2), kv_heads=G, dim=pick(4, 10, 16, 24, 36, 64), vdim=pick(6, 16, 20, 33, 64), conv=pick(1, 2, 3, 4, 5), **kw)
    layers = []
    for _ in range(int(r.integers(1, 6))):
        if pick(0, 1):
            layers.append(layer({"type": "delta", "mixer": some_rule()}, pick(0, 12, 30, 64)))
        else:
            G = pick(1, 2, 3)
            d = pick(8, 18, 32, 40, 64)
            rot = yarn(dims=min(d, pick(2, 8, 16, 64)), base=float(pick(100.0, 10000.0, 1e6)), scaling=pick(True, False), factor=float(pick(1.0, 2.0, 8.0)), original=pick(32, 100, 4000),
                       fast=float(pick(4.0, 32.0)), slow=float(pick(1.0, 0.5)))
            layers.append(layer(parallel(heads=G * pick(1, 2, 4), kv_heads=G, dim=d, vdim=pick(8, 20, 24, 64, 128), conv=pick(1, 2, 3, 4, 6), size=pick(0, 1, 5, 31, 32, 33, 64, 100),
                                         keep=pick(0, 1, 4, 32, 33, 64), rot=rot, scale=float(pick(0.1, 0.3, 0.6)), left_scale=float(pick(0.3, 1.0)), right_scale=float(pick(0.5, 1.0, 1.5)),
                                         right=some_rule(a_rank=pick(1, 7, 24, 40), g_rank=pick(1, 8, 24, 33))), pick(0, 12, 30, 64)))
    return config(layers, width=pick(72, 96, 120, 160), vocab=pick(90, 211, 300), eps=float(pick(1e-6, 1e-5)), mult=float(pick(0.4, 1.0)), side=pick(4, 8, 24, 33))


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(10))
def test_random_layer_lists(seed):
    cfg = random_config(100 + seed)
    r = np.random.default_rng(seed)
    ids, other = tokens(150, cfg["vocab"], 200 + seed), tokens(70, cfg["vocab"], 300 + seed)
    for precision, tol in (("f32", F32_TOL), ("split", SPLIT_TOL)):
        m, w = make(cfg, 400 + seed, precision=precision)
        want, want2 = oracle_logits(cfg, w, ids), oracle_logits(cfg, w, other)
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

    def refused(change, layer_list=(0, 1)):
        cfg = config([layer(delta()), layer(parallel())])
        change(cfg)
        with pytest.raises(crane_b200.CraneB200Error):
            crane_b200.SuvapelModel(cfg, device=0, max_tokens=256).close()
    refused(lambda c: c["layers"][0].update(type="other"))
    refused(lambda c: c["layers"][0]["mixer"].update(heads=3, kv_heads=2))
    refused(lambda c: c["layers"][1]["mixer"].pop("right"))
    refused(lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26))
    refused(lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=-1))
    refused(lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0))
    refused(lambda c: c["layers"][1]["mlp"].update(kind="moe"))
    cfg = config([layer(parallel())])
    w = O.random_weights(cfg, 1)
    m = crane_b200.SuvapelModel(cfg, device=0, max_tokens=256)
    t = lambda k: w[k].to(torch.float32).numpy()
    m.load_tensor("l0.mix.right.a1", t("l0.mix.right.a1"))
    with pytest.raises(crane_b200.CraneB200Error):
        m.load_tensor("l0.mix.right.a2", np.zeros((48, 5), np.float32))       # another rank than its partner's
    with pytest.raises(crane_b200.CraneB200Error):
        m.load_tensor("l0.mix.right.extra", t("l0.mix.right.b"))
    with pytest.raises(crane_b200.CraneB200Error):
        m.finalize()
    m.close()


@pytest.mark.gpu
def test_model_folder_loader_and_trace_runner(tmp_path):
    import json, os, subprocess, sys
    cfg = copy.deepcopy(FULL)
    for lc in cfg["layers"]:                                    # ranks come with their tensors, not with config.json
        for k in ("a_rank", "g_rank"):
            lc["mixer"].get("right", {}).pop(k, None)
    w = O.random_weights(FULL, 23)
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
    wa, wb = oracle_logits(FULL, w, a), oracle_logits(FULL, w, b)
    read = lambda n: np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    assert rel(read(0), wa[49:50]) < F32_TOL
    assert rel(read(1), np.stack([wb[2], wb[69], wa[50]])) < F32_TOL
    assert not (out / "2.f32").exists()
    assert rel(read(3), wb[69:70]) < F32_TOL                    # request c runs on the slot and pages b gave back
