"""GPU tests of the Tegolix design on the layer-list path: the CUDA backend (forward / sessions / decode_greedy behind
arch.load_model) against the plain numpy oracle in tests/_tegolix_ref.py, on small random models made here.

float32 mode is compared tightly with the oracle; bfloat16 mode loosely with the oracle."""
import json
import os
import subprocess

import numpy as np
import pytest

from powerserve_b200 import arch, arch_synth, capi
from tests import _tegolix_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GL, PA = arch_synth.tegolix_gla_layer, arch_synth.tegolix_parallel_layer
YARN = {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 1.0}
# every mixer and feed-forward, unequal head counts and sizes
MIXED = [PA(4, 2, 10, 14, window=21, rwkv=(3, 12), rot_dims=6, rot_base=300.0, scaling=YARN, softcap=4.0, ff=24, experts=5, top=3, identity=2, shared_ff=40),
         GL(3, 12, 10, tau=6.0, ff=56), PA(3, 3, 8, 6, window=33, rwkv=(2, 9), left_scale=1.1, right_scale=0.7, ff=30), GL(2, 20, 7, tau=1.0, ff=16, experts=6, top=2)]


def make(tmp_path, layers, width=48, vocab=96, seed=0, eps=1e-6, edit=None, name="m", side_dim=10, rank=6):
    cfg = arch_synth.tegolix_config(width, vocab, layers, side_dim=side_dim, eps=eps)
    t = arch_synth.tegolix_weights(cfg, seed=seed, rank=rank)
    if edit:
        edit(t)
        t = {k: R.bf16_round(v) for k, v in t.items()}
    d = str(tmp_path / name)
    arch_synth.write_model_dir(d, cfg, t)
    return d, cfg, t


def tokens(vocab, n, seed=0):
    return [int(v) for v in np.random.default_rng(seed).integers(0, vocab, n)]


def run(model, toks, cuts=None):
    """logits of every position, the sequence fed in portions of the given sizes (cycled); None = one portion per batch cap"""
    model.reset()
    cap, out, lo, k = model.desc.max_batch, [], 0, 0
    while lo < len(toks):
        s = min(cap if cuts is None else min(cuts[k % len(cuts)], cap), len(toks) - lo)
        out.append(model.forward(toks[lo:lo + s]))
        lo, k = lo + s, k + 1
    return np.concatenate(out)


def rel_err(got, ref):
    """per position: rms of the difference over rms of the reference"""
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.maximum(np.sqrt((ref ** 2).mean(-1)), 1e-6)


TOL = {"float32": 4e-5, "bfloat16": 6e-2}


def check(got, ref, dtype, what=""):
    e = rel_err(got, ref)
    assert e.max() < TOL[dtype], f"{what}: worst relative error {e.max():.3g} at position {int(e.argmax())} ({dtype})"
    if dtype == "bfloat16":
        assert np.median(e) < 2e-2, f"{what}: median relative error {np.median(e):.3g}"


def check_routed_bf16(got, ref, what=""):
    """models with a router: a position whose choice is a close call may flip under rounding, so a few positions may be far off"""
    e = rel_err(got, ref)
    assert np.median(e) < 2e-2 and np.mean(e > TOL["bfloat16"]) < 0.1, f"{what}: median {np.median(e):.3g}, {np.mean(e > TOL['bfloat16']):.3g} of the positions over"


def both_paths(d, toks, ref, what, n_ctx, cap=64, cuts=([7, 2, 33, 1],), decode_from=None):
    """float32: portions of the batch cap, ragged portions, and the tail decoded token by token, all against the oracle"""
    m = arch.load_model(d, dtype="float32", max_batch=cap, n_ctx=n_ctx)
    check(run(m, toks), ref, "float32", what + ", portions of the batch cap")
    for c in cuts:
        check(run(m, toks, list(c)), ref, "float32", what + f", portions {list(c)}")
    k = decode_from if decode_from is not None else len(toks) // 2
    m.reset()
    for lo in range(0, k, cap):
        m.forward(toks[lo:min(k, lo + cap)], lm_head=False)
    dec = np.concatenate([m.forward(toks[i:i + 1]) for i in range(k, len(toks))])
    check(dec, ref[k:], "float32", what + ", decoded alone")
    m.close()


def alone(tmp_path, layer, what, seed, n=45, width=48, n_ctx=64, moved=(), **kw):
    """one layer by itself, its residual stream too; `moved`: (tensor, value) pairs that must show in the oracle's logits"""
    d, cfg, t = make(tmp_path, [layer], seed=seed, width=width, **kw)
    toks = tokens(96, n, seed)
    taps = []
    ref = R.forward(cfg, t, toks, taps=taps)
    for name, new in moved:
        t2 = dict(t)
        t2[name] = np.full_like(t[name], new)
        assert rel_err(R.forward(cfg, t2, toks), ref).max() > 5e-3, name
    m = arch.load_model(d, dtype="float32", max_batch=64, n_ctx=n_ctx)
    m.be.set_option("arch_taps", 1)
    check(run(m, toks), ref, "float32", what)
    check(m.layer_tap(0, len(toks)), taps[0], "float32", "residual after the layer")
    m.close()
    both_paths(d, toks, ref, what, n_ctx, cuts=([7, 2, 33, 1], [2]))


# ------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("heads,dim,vdim,tau,rank", [(3, 12, 10, 6.0, 6), (1, 16, 64, 16.0, 16), (2, 40, 7, 1.0, 3), (4, 8, 130, 30.0, 8), (5, 1, 3, 2.0, 1), (2, 100, 24, 16.0, 24), (1, 200, 33, 4.0, 9)])
def test_gated_linear_attention_alone(tmp_path, heads, dim, vdim, tau, rank):
    alone(tmp_path, GL(heads, dim, vdim, tau=tau), "gated linear attention", 1, rank=rank, moved=[("l0.mix.a2.b", -6.0), ("l0.mix.g", 0.0), ("l0.mix.a2", 0.0)])


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,rwkv", [(4, 2, 10, 14, 6, (3, 12)), (3, 3, 8, 8, 8, (1, 16)), (6, 1, 12, 4, 2, (4, 5)), (1, 1, 6, 20, 4, (2, 40)), (8, 4, 16, 130, 16, (2, 64)),
                                                              (2, 1, 4, 2, 4, (5, 1)), (2, 2, 70, 66, 70, (1, 130))])
def test_attention_beside_time_mixing(tmp_path, heads, kv_heads, dim, vdim, rot, rwkv):
    alone(tmp_path, PA(heads, kv_heads, dim, vdim, window=17, rwkv=rwkv, rot_dims=rot, rot_base=50.0, scaling=YARN, softcap=3.0), "attention beside a time mixing", 2,
          moved=[("l0.mix.left.g", 0.0), ("l0.mix.left.q.norm", 0.3), ("l0.mix.left.k.norm", 0.3), ("l0.mix.left.o", 0.0), ("l0.mix.right.o", 0.0), ("l0.mix.right.u", 4.0), ("l0.mix.right.mu.r", 0.0),
                 ("l0.mix.right.mu.k", 0.0), ("l0.mix.right.mu.v", 0.0), ("l0.mix.right.mu.g", 0.0), ("l0.mix.right.w0", 1.5), ("l0.mix.right.norm", 0.3)])


def test_the_mixture_of_the_decay_input(tmp_path):
    """a strong low-rank term, so that the decay's own mixture and its tanh show"""
    def edit(t):
        t["l0.mix.right.w2"] = t["l0.mix.right.w2"] * 3.0
        t["l0.mix.right.w0"] = np.full_like(t["l0.mix.right.w0"], -1.0)
    alone(tmp_path, PA(1, 1, 4, 4, window=3, rwkv=(3, 8), left_scale=0.1, right_scale=2.0), "decay of the time mixing", 3, edit=edit, moved=[("l0.mix.right.mu.w", 0.0), ("l0.mix.right.w1", 0.0)])


@pytest.mark.parametrize("scaling,softcap,left,right", [(None, None, 1.0, 1.0), (YARN, 0.7, 0.3, 1.9), ({"factor": 8.0, "original": 16, "fast": 2.0, "slow": 1.0}, 20.0, 2.0, 0.2)])
def test_constants_of_the_parallel_mixer(tmp_path, scaling, softcap, left, right):
    def edit(t):
        t["l0.mix.left.q.norm"] = t["l0.mix.left.q.norm"] * 2.0
    layer = PA(4, 2, 12, 8, window=30, rwkv=(2, 6), rot_base=20.0, scaling=scaling, softcap=softcap, left_scale=left, right_scale=right, scale=0.4)
    d, cfg, t = make(tmp_path, [layer], seed=4, edit=edit)
    toks = tokens(96, 60, 4)
    ref = R.forward(cfg, t, toks)
    for key, other in (("left_scale", left + 0.3), ("right_scale", right + 0.3)):
        c2 = json.loads(json.dumps(cfg))
        c2["layers"][0]["mixer"][key] = other
        assert rel_err(R.forward(c2, t, toks), ref).max() > 1e-2, key
    if softcap and softcap < 5:
        c2 = json.loads(json.dumps(cfg))
        c2["layers"][0]["mixer"]["left"]["softcap"] = 2 * softcap
        assert rel_err(R.forward(c2, t, toks), ref).max() > 3e-3
    both_paths(d, toks, ref, "constants", 64, cuts=([2], [9, 64]))


def test_dense_feed_forward_alone(tmp_path):
    alone(tmp_path, GL(1, 2, 2, ff=72), "relu feed-forward", 5, moved=[("l0.mlp.up", 0.0), ("l0.ls2", 0.0), ("l0.norm2b", 1.0)])


@pytest.mark.parametrize("experts,top,identity,ff,shared", [(5, 2, 2, 24, 40), (16, 3, 0, 20, 12), (3, 3, 1, 17, 9), (1, 1, 0, 8, 0), (1, 4, 6, 8, 0), (40, 5, 9, 12, 0), (130, 4, 30, 8, 16), (2, 1, 40, 8, 5), (2, 5, 3, 200, 24)])
def test_routed_feed_forward_alone(tmp_path, experts, top, identity, ff, shared):
    alone(tmp_path, GL(1, 2, 2, ff=ff, experts=experts, top=top, identity=identity, shared_ff=shared), "routed experts", 6,
          moved=([("l0.mlp.shared.down", 0.0), ("l0.mlp.shared.sg", 0.0)] if shared else []) + ([("l0.mlp.correction", 0.0)] if top < experts + identity and experts < 100 else []))


def test_corrections_choose_but_do_not_weigh(tmp_path):
    """corrections that are all negative, and one that always wins with a small score"""
    def edit(t):
        c = np.full_like(t["l0.mlp.correction"], -2.0)
        c[3], c[5] = -0.5, -0.75                                     # an expert and an identity output, always these two
        t["l0.mlp.correction"] = c
    alone(tmp_path, GL(1, 2, 2, ff=16, experts=5, top=2, identity=2), "corrections", 7, edit=edit, moved=[("l0.mlp.correction", 0.0)])


@pytest.mark.parametrize("side_dim", [1, 10, 33, 96])
def test_token_input_alone(tmp_path, side_dim):
    alone(tmp_path, GL(1, 2, 2), "token input", 8, side_dim=side_dim, moved=[("l0.side.gate", 0.0), ("l0.side.norm", 0.0), ("side.embed", 0.5)])


def test_token_input_takes_its_own_layers_part(tmp_path):
    layers = [GL(1, 2, 2), PA(1, 1, 4, 4, window=4, rwkv=(1, 2)), GL(1, 2, 2, ff=6)]
    d, cfg, t = make(tmp_path, layers, seed=9, side_dim=7)
    toks = tokens(96, 30, 9)
    taps = []
    ref = R.forward(cfg, t, toks, taps)
    m = arch.load_model(d, dtype="float32", max_batch=32, n_ctx=32)
    m.be.set_option("arch_taps", 1)
    check(run(m, toks), ref, "float32", "three layers")
    for i in range(3):
        check(m.layer_tap(i, 30), taps[i], "float32", f"residual after layer {i}")
    m.close()
    both_paths(d, toks, ref, "three layers", 32)


# ------------------------------------------------------------------------------------------------- window edges, far keys, the start
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 63, 64, 65, 130])
def test_window_edges(tmp_path, window):
    """one key stands out (a token that occurs once, which every query asks for): one token too many or too few in the window shows at full size"""
    def edit(t):
        t["l0.mix.left.k"] = t["l0.mix.left.k"] * 0
        t["l0.mix.left.k"][4, 0] = 8.0                                # the key lies along one axis by the first input channel; the rotated pair
        t["l0.mix.left.q"] = t["l0.mix.left.q"] * 0                   # stays empty, so the score does not depend on distance
        t["l0.mix.left.q"][:, 1] = 4.0                                # the second input channel is the same for every token
        t["l0.mix.left.q.norm"], t["l0.mix.left.k.norm"] = t["l0.mix.left.q.norm"] * 0 + 3.0, t["l0.mix.left.k.norm"] * 0 + 3.0
        t["embed"][:, 0], t["embed"][:, 1] = -6.0, 6.0
        t["embed"][0, 0] = 6.0
        t["l0.norm1"] = t["l0.norm1"] * 0
    at = 9
    layer = PA(1, 1, 8, 8, window=window, rwkv=(1, 4), rot_dims=2, softcap=80.0, scale=1.0, left_scale=2.0, right_scale=0.1)
    n = at + window + 40
    d, cfg, t = make(tmp_path, [layer], seed=10, width=32, vocab=40, edit=edit)
    toks = [1 + v % 39 for v in tokens(39, n, 10)]
    toks[at] = 0
    ref = R.forward(cfg, t, toks)
    c2 = json.loads(json.dumps(cfg))
    for other, where in ((window + 1, at + window), (max(window - 1, 1), at + window - 1)):
        if other != window:
            c2["layers"][0]["mixer"]["left"]["mask"]["size"] = other
            assert rel_err(R.forward(c2, t, toks), ref)[where] > 5e-2, (window, other)
    for start in (0, 50):                                             # the edge inside a batch tile and further on
        tk = [1 + v % 39 for v in tokens(39, start, 11)] + toks
        both_paths(d, tk, R.forward(cfg, t, tk), f"window {window}", -(-len(tk) // 16) * 16, cap=128, cuts=([2], [window + 1, 3], [31, 64]), decode_from=start + at - 1)


@pytest.mark.parametrize("kind", ["gla", "rwkv"])
def test_state_reaches_across_portions(tmp_path, kind):
    """slow decays: the first token still shows in the last logits, through every cut"""
    def edit(t):
        if kind == "gla":
            t["l0.mix.a2.b"] = np.full_like(t["l0.mix.a2.b"], 9.0)
        else:
            t["l0.mix.right.w0"] = np.full_like(t["l0.mix.right.w0"], -8.0)
            t["l0.mix.left.o"] = t["l0.mix.left.o"] * 0
        t["embed"][0] = 8.0 * np.sign(t["embed"][1])
    layer = GL(2, 8, 8, tau=16.0) if kind == "gla" else PA(1, 1, 4, 4, window=3, rwkv=(2, 8))
    d, cfg, t = make(tmp_path, [layer], seed=12, width=32, edit=edit)
    toks = [0] + [1 + v % 95 for v in tokens(95, 199, 12)]
    ref = R.forward(cfg, t, toks)
    assert rel_err(R.forward(cfg, t, [7] + toks[1:])[-1:], ref[-1:]).max() > 1e-3
    both_paths(d, toks, ref, "state", 208, cap=96, cuts=([2], [3, 1, 4], [32], [33, 31]), decode_from=40)


@pytest.mark.parametrize("value", [-30.0, -4.0, 0.0, 30.0])
def test_decays_from_nearly_one_to_nearly_zero(tmp_path, value):
    def edit(t):
        for k in ("l0.mix.a2.b", "l1.mix.right.w0"):
            t[k] = np.full_like(t[k], value if k[1] == "0" else {-30.0: 3.0, -4.0: 0.0, 0.0: -4.0, 30.0: -30.0}[value])
    layers = [GL(2, 8, 8, tau=2.0), PA(1, 1, 4, 4, window=3, rwkv=(2, 8))]
    d, cfg, t = make(tmp_path, layers, seed=13, width=32, edit=edit)
    toks = tokens(96, 90, 13)
    both_paths(d, toks, R.forward(cfg, t, toks), f"decay bias {value}", 96)


def test_rotation_far_from_the_start(tmp_path):
    """a base that leaves every pair turning fast: the angle's error would show first at the last positions"""
    def edit(t):
        t["l0.mix.left.q.norm"] = t["l0.mix.left.q.norm"] * 2.0
    d, cfg, t = make(tmp_path, [PA(2, 1, 16, 12, window=40, rwkv=(1, 4), rot_base=3.0)], seed=14, width=32, edit=edit)
    toks = tokens(96, 900, 14)
    both_paths(d, toks, R.forward(cfg, t, toks), "rotation", 912, cap=256, cuts=([200, 3],), decode_from=880)


def test_the_first_tokens(tmp_path):
    """the first tokens of a sequence on a set that a longer sequence has used: nothing of it may show (keys, state, the token before)"""
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=15)
    m = arch.load_model(d, dtype="float32", max_batch=64, n_ctx=64)
    for n in (60, 59):
        long_, short = tokens(130, n, 15), tokens(130, 6, 16)
        ref = R.forward(cfg, t, short)
        for cuts in ([1], [2], [6], [3, 1]):
            run(m, long_)
            check(run(m, short, cuts), ref, "float32", f"first tokens, portions {cuts}")
    m.close()


# ------------------------------------------------------------------------------------------------- schedules
def test_whole_prompt_portions_and_decoding_agree_in_both_precisions(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=17)
    toks = tokens(130, 150, 17)
    ref = R.forward(cfg, t, toks)
    both_paths(d, toks, ref, "mixed model", 160, cap=64, cuts=([7, 2, 33, 1], [2], [64, 3]))
    m = arch.load_model(d, dtype="bfloat16", max_batch=64, n_ctx=160)
    whole = run(m, toks)
    check_routed_bf16(whole, ref, "whole prompt")
    for cuts in ([1], [2], [5, 40, 3]):
        got = run(m, toks, cuts)
        check_routed_bf16(got, ref, f"portions {cuts}")
        assert np.median(rel_err(got, whole)) < 2e-2
    m.close()


def test_bfloat16_without_a_router(tmp_path):
    layers = [PA(4, 2, 16, 8, window=30, rwkv=(4, 16), scaling=YARN, ff=64), GL(4, 24, 16, ff=64), GL(2, 8, 40)]
    d, cfg, t = make(tmp_path, layers, width=64, vocab=120, seed=18)
    toks = tokens(120, 150, 18)
    ref = R.forward(cfg, t, toks)
    m = arch.load_model(d, dtype="bfloat16", max_batch=64, n_ctx=160)
    for cuts in (None, [1], [2, 50]):
        check(run(m, toks, cuts), ref, "bfloat16", f"portions {cuts}")
    m.close()


def test_single_token_kernels_match_the_batch_kernels(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=19)
    toks = tokens(130, 100, 19)
    for dtype in ("float32", "bfloat16"):
        m = arch.load_model(d, dtype=dtype, max_batch=32, n_ctx=112)
        a = run(m, toks, [1])
        m.be.set_option("arch_simple", 1)
        b = run(m, toks, [1])
        assert np.median(rel_err(a, b)) < (1e-5 if dtype == "float32" else 2e-2), dtype
        if dtype == "float32":
            assert rel_err(a, b).max() < 8e-5
        m.close()


def test_replayed_step_matches_the_plain_launches(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=20)
    toks = tokens(130, 90, 20)
    for dtype in ("float32", "bfloat16"):
        m = arch.load_model(d, dtype=dtype, max_batch=40, n_ctx=96)
        g0 = m.be.counter("graph_replays")
        a = run(m, toks, [1])
        assert m.be.counter("graph_replays") - g0 == len(toks)
        m.reset()
        m.forward(toks[:40], lm_head=False)
        ids_a = list(m.decode_greedy(toks[40], 20))
        m.be.set_option("graph", 0)
        b = run(m, toks, [1])
        m.reset()
        m.forward(toks[:40], lm_head=False)
        ids_b = list(m.decode_greedy(toks[40], 20))
        np.testing.assert_array_equal(a, b)                         # the same kernels on the same data
        assert ids_a == ids_b
        m.be.set_option("graph", 1)
        for opt in ("arch_pdl", "arch_fork"):
            m.be.set_option(opt, 0)
            np.testing.assert_array_equal(run(m, toks, [1]), a)
            m.be.set_option(opt, 1)
        m.close()


def test_tensor_core_gemm_matches_the_tile_kernels(tmp_path):
    """bfloat16 batches: the tcgen05 GEMM (six operand sets in one product, the token input's table row, experts) against the fp32-FMA tiles"""
    layers = [PA(6, 3, 24, 40, window=90, rwkv=(5, 40), scaling=YARN, ff=200), GL(4, 30, 36, ff=136), PA(1, 1, 130, 8, window=9, rwkv=(1, 3))]
    d, cfg, t = make(tmp_path, layers, width=136, vocab=300, seed=21, side_dim=150, rank=20)
    toks = tokens(300, 300, 21)
    m = arch.load_model(d, dtype="bfloat16", max_batch=160, n_ctx=304)
    n0 = m.be.counter("kernel_launches")
    a = run(m, toks)
    n1 = m.be.counter("kernel_launches")
    m.be.set_option("arch_tc", 0)
    b = run(m, toks)
    assert n1 > n0
    e = rel_err(a, b)
    assert np.median(e) < 1e-2 and e.max() < 4e-2, (np.median(e), e.max())
    check(a, R.forward(cfg, t, toks), "bfloat16", "tensor-core path against the oracle")
    m.close()
    d, cfg, t = make(tmp_path, [GL(2, 24, 40, ff=200, experts=7, top=3, identity=2, shared_ff=130)], width=136, vocab=300, seed=22, name="moe")
    m = arch.load_model(d, dtype="bfloat16", max_batch=160, n_ctx=304)
    a = run(m, toks)
    m.be.set_option("arch_tc", 0)
    b = run(m, toks)
    e = rel_err(a, b)
    assert np.median(e) < 1e-2 and np.mean(e > 4e-2) < 0.02, (np.median(e), e.max())
    check_routed_bf16(a, R.forward(cfg, t, toks), "experts on the tensor cores")
    m.close()


def test_scan_options_agree(tmp_path):
    """one or two value columns per lane of the recurrence's scan: the same numbers"""
    d, cfg, t = make(tmp_path, [GL(2, 40, 70), PA(1, 1, 4, 4, window=5, rwkv=(2, 60))], seed=23)
    toks = tokens(96, 70, 23)
    m = arch.load_model(d, dtype="float32", max_batch=64, n_ctx=80)
    m.be.set_option("arch_scan_nc", 1)
    a = run(m, toks)
    m.be.set_option("arch_scan_nc", 2)
    np.testing.assert_array_equal(a, run(m, toks))
    m.close()


def test_sessions_interleaved_and_sets_reused(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=24)
    reqs = [tokens(130, n, 40 + i) for i, n in enumerate((50, 9, 33, 64))]
    refs = [R.forward(cfg, t, r) for r in reqs]
    m = arch.load_model(d, dtype="float32", max_batch=16, n_ctx=64)
    sid = [m.session_create() for _ in range(3)]
    got = [[] for _ in reqs]
    at = [0, 0, 0, 0]
    sizes = [5, 2, 16, 1, 7]
    live, k = [0, 1, 2], 0
    while live:
        for r in list(live):
            s = min(sizes[k % len(sizes)], len(reqs[r]) - at[r])
            k += 1
            m.session_select(sid[r])
            assert m.position == at[r]
            got[r].append(m.forward(reqs[r][at[r]:at[r] + s]))
            at[r] += s
            if at[r] == len(reqs[r]):
                live.remove(r)
                if r == 1:              # the short request ends first: its set is freed and a new request takes a new one
                    m.session_select(0)
                    m.session_destroy(sid[1])
                    sid.append(m.session_create())
                    live.append(3)
    for r in range(4):
        check(np.concatenate(got[r]), refs[r], "float32", f"request {r} among others")
    # the same set used again from position 0: the recurrent state of the longer request must not leak
    m.session_select(sid[0])
    m.reset()
    check(run(m, reqs[2], [16]), refs[2], "float32", "set reused after reset")
    check(run(m, reqs[1], [1]), refs[1], "float32", "set reused once more, token by token")
    m.reset()
    m.forward(reqs[2][:16])
    with pytest.raises(capi.PsCudaError):                           # recurrent state cannot be cut back, only to the start
        m.be.kv_rollback(13)
    m.be.kv_rollback(16)
    assert m.position == 0
    check(m.forward(reqs[2][:16]), refs[2][:16], "float32", "from the start after a rollback to 0")
    m.close()


def test_long_decoding(tmp_path):
    layers = [PA(4, 1, 8, 12, window=100, rwkv=(2, 8), ff=16), GL(2, 12, 8, ff=16, experts=4, top=2, identity=1)]
    d, cfg, t = make(tmp_path, layers, width=32, vocab=50, seed=25)
    toks = tokens(50, 400, 25)
    ref = R.forward(cfg, t, toks)
    for dtype in ("float32", "bfloat16"):
        m = arch.load_model(d, dtype=dtype, max_batch=8, n_ctx=400)
        m.reset()
        m.forward(toks[:6], lm_head=False)
        dec = np.concatenate([m.forward(toks[i:i + 1]) for i in range(6, 400)])
        if dtype == "float32":
            check(dec, ref[6:], dtype, "394 tokens decoded alone")
        else:
            check_routed_bf16(dec, ref[6:], "394 tokens decoded alone")
        m.close()


@pytest.mark.parametrize("layers,width,vocab,side,rank", [
    ([GL(1, 1, 1)], 8, 11, 1, 1),                                                                    # the smallest of everything
    ([PA(1, 1, 2, 2, window=1, rwkv=(1, 1), ff=1)], 8, 11, 3, 1),
    ([PA(8, 8, 8, 8, window=20, rwkv=(2, 8), ff=8)], 40, 64, 4, 2),                                  # no key sharing
    ([PA(12, 1, 12, 20, window=7, rwkv=(1, 30), ff=20, experts=2, top=1, shared_ff=7)], 56, 77, 9, 16),   # one shared key head
    ([GL(5, 7, 9, ff=37), PA(5, 5, 6, 10, window=11, rwkv=(3, 7), rot_dims=4, ff=11, experts=3, top=2), GL(3, 3, 5)], 50, 101, 7, 5),   # nothing a multiple of four
    ([PA(16, 4, 32, 64, window=64, rwkv=(8, 32), scaling=YARN, ff=96, experts=8, top=2, shared_ff=64), GL(4, 64, 128, ff=96)], 128, 300, 32, 32),
    ([GL(1, 256, 20), PA(2, 1, 100, 90, window=33, rwkv=(1, 256))], 96, 60, 5, 8),                   # the widest states
    ([PA(64, 2, 4, 4, window=16, rwkv=(4, 4))], 32, 60, 6, 4),                                       # many heads
    ([GL(2, 8, 8), GL(4, 4, 4), PA(2, 2, 8, 8, window=40, rwkv=(2, 4))], 32, 60, 3, 3),              # no feed-forward anywhere
])
def test_other_sizes(tmp_path, layers, width, vocab, side, rank):
    d, cfg, t = make(tmp_path, layers, width=width, vocab=vocab, seed=26, eps=3e-6, side_dim=side, rank=rank)
    toks = tokens(vocab, 75, 26)
    ref = R.forward(cfg, t, toks)
    m = arch.load_model(d, dtype="float32", max_batch=32, n_ctx=80)
    check(run(m, toks), ref, "float32", "portions of 32")
    check(run(m, toks, [2, 31, 1]), ref, "float32", "ragged portions")
    check(run(m, toks[:40], [1]), ref[:40], "float32", "token by token")
    m.close()
    m = arch.load_model(d, dtype="bfloat16", max_batch=80, n_ctx=80)
    check_routed_bf16(run(m, toks), ref, "whole prompt")
    m.close()


def test_odd_cache_length(tmp_path):
    """a cache length that is no multiple of four: no bulk copies of value rows, the state behind the K rows still aligned"""
    d, cfg, t = make(tmp_path, [PA(2, 1, 6, 6, window=9, rwkv=(2, 5))], seed=27)
    toks = tokens(96, 37, 27)
    both_paths(d, toks, R.forward(cfg, t, toks), "odd cache", 37, cap=16)


# ------------------------------------------------------------------------------------------------- entry points
def test_greedy_generation_through_the_entry_points(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=28)
    prompt = tokens(130, 21, 28)
    m = arch.load_model(d, dtype="float32", max_batch=8, n_ctx=64)
    ids, lg = m.generate(prompt, 12, batch_size=8)                  # prefill in portions + one forward per token
    m.reset()
    m.prefill(prompt, 8)
    ids2 = [int(v) for v in m.decode_greedy(prompt[-1], 12)]        # the device-side greedy loop
    assert ids == ids2
    assert m.position == len(prompt) - 1 + 12
    seq = list(prompt)
    for step, tok in enumerate(ids):
        ref = R.forward(cfg, t, seq)[-1]
        assert rel_err(lg[step][None], ref[None]).max() < 4e-5
        assert ref[tok] >= ref.max() - 1e-4 * np.abs(ref).max()
        seq.append(tok)
    m.forward_lazy([seq[-1]])
    vals, idx = m.sample_topk(5)
    full = R.forward(cfg, t, seq)[-1]
    assert list(idx) == [int(v) for v in np.argsort(-full, kind="stable")[:5]]
    m.close()


def test_bad_configurations_are_refused(tmp_path):
    odd = PA(2, 1, 8, 8, window=4, rwkv=(1, 4), rot_dims=5)         # an odd number of rotated dimensions
    for i, layers in enumerate([[PA(3, 2, 8, 8, window=4, rwkv=(1, 4))], [odd], [PA(2, 1, 8, 7, window=4, rwkv=(1, 4))], [GL(1, 300, 4)], [GL(1, 4, 4, ff=8, experts=2, top=4, identity=1)]]):
        cfg = arch_synth.tegolix_config(32, 40, layers, side_dim=4)
        arch_synth.write_model_dir(str(tmp_path / f"bad{i}"), cfg, arch_synth.tegolix_weights(cfg, seed=29))
        with pytest.raises(capi.PsCudaError):
            arch.load_model(str(tmp_path / f"bad{i}"), dtype="float32", max_batch=8, n_ctx=16)


def test_trace_runner_and_generation_command_lines(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=30)
    a, b = tokens(130, 40, 30), tokens(130, 17, 31)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:], "want": [7, 3]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [16]}], "end": ["b"]}]
    out = tmp_path / "out"
    ra, rb = R.forward(cfg, t, a), R.forward(cfg, t, b)
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out), "--max-tokens", "40", "--max-batch", "16"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    check(np.fromfile(out / "0.f32", "<f4").reshape(2, 130), ra[[0, 29]], "float32", "step 0")
    assert not (out / "1.f32").exists()
    check(np.fromfile(out / "2.f32", "<f4").reshape(2, 130), ra[[39, 35]], "float32", "step 2 (order of `want`)")
    check(np.fromfile(out / "3.f32", "<f4").reshape(1, 130), rb[[16]], "float32", "step 3")
    prompt = tokens(130, 19, 29)
    exe = os.path.join(ROOT, "bin", "ps_generate")
    p = subprocess.run([exe, "--model", d, "--dtype", "float32", "--ids", " ".join(map(str, prompt)), "--n", "10", "--prefill-batch", "8"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    ids = json.loads(p.stdout.strip().splitlines()[-1])["ids"]
    m = arch.load_model(d, dtype="float32", max_batch=32, n_ctx=32)
    want, _ = m.generate(prompt, 10, batch_size=8)
    assert ids == want
    m.close()
