"""CPU-only checks around the Tegolix design: the registry's reading of a configuration (every size and constant comes from the file or a
stored tensor's shape), the tensor names, the exported rotation table, and the oracle's own invariants (it is what the GPU tests
compare with, so it is checked against hand-computed cases and second formulations here)."""
import json
import math

import numpy as np
import pytest

from powerserve_b200 import arch, arch_synth, capi
from tests import _tegolix_ref as R

GL, PA = arch_synth.tegolix_gla_layer, arch_synth.tegolix_parallel_layer
DESCRIBE, NAMES = arch.ARCHITECTURES["Tegolix"]
YARN = {"factor": 3.0, "original": 40, "fast": 16.0, "slow": 2.0}


class Shape:
    def __init__(self, *s):
        self.shape = s


def test_registry_reads_every_size_from_the_configuration():
    layers = [PA(6, 3, 14, 10, window=23, rwkv=(5, 7), rot_dims=8, rot_base=777.0, scaling=YARN, softcap=31.0, scale=0.21, left_scale=0.4, right_scale=1.7, ff=26),
              GL(3, 9, 11, tau=5.0, ff=18, experts=7, top=4, identity=3, shared_ff=21), GL(2, 4, 6, tau=1.0), PA(2, 2, 8, 4, window=5, rwkv=(1, 3), softcap=None, ff=12, experts=4)]
    cfg = arch_synth.tegolix_config(60, 99, layers, side_dim=13, eps=3e-5)
    descs, top = DESCRIBE(cfg, {"l0.mix.right.w1": Shape(17, 60), "l1.mix.a1": Shape(19, 60), "l2.mix.a1": Shape(1, 60), "l3.mix.right.w1": Shape(2, 60)})
    assert top == {"dim": 60, "vocab_size": 99, "norm_eps": 3e-5, "embed_scale": 1.0, "norm_unit_offset": 1, "token_dim": 13, "token_slots": 4}
    assert [d.token_slot for d in descs] == [1, 2, 3, 4]
    assert all(d.block_kind == capi.BLOCK_SEQUENTIAL and d.post_norm == 1 and d.layer_scale == 1 and d.raw_input == 0 for d in descs)
    d = descs[0]
    assert (d.mixer_kind, d.n_heads, d.n_kv_heads, d.qk_dim, d.v_dim, d.window) == (capi.MIXER_ATTENTION, 6, 3, 14, 10, 23)
    assert (d.rope_dims, d.rope_base, d.rope_factor, d.rope_original, d.rope_fast, d.rope_slow, d.rope_interleaved) == (8, 777.0, 3.0, 40, 16.0, 2.0, 0)
    assert (d.score_softcap, d.v_rope, d.qk_norm, d.out_gate) == (31.0, 1, capi.QKNORM_HEAD_W, capi.GATE_HEAD) and abs(d.score_scale - 0.21) < 1e-7
    assert (d.side_kind, d.side_heads, d.side_width, d.decay_rank) == (capi.MIXER_RWKV, 5, 35, 17)
    assert abs(d.mix_scale - 0.4) < 1e-7 and abs(d.side_scale - 1.7) < 1e-7
    assert (d.mlp_kind, d.expert_ff, d.act_kind, d.mlp_ungated) == (capi.MLP_DENSE, 26, capi.ACT_RELU, 0)
    d = descs[1]
    assert (d.mixer_kind, d.n_heads, d.qk_dim, d.v_dim, d.decay_tau, d.decay_rank, d.rope_dims, d.window) == (capi.MIXER_GLA, 3, 9, 11, 5.0, 19, 0, 0)
    assert (d.mlp_kind, d.n_experts, d.top_k, d.expert_ff, d.route_identity, d.shared_ff, d.shared_gate) == (capi.MLP_ROUTED, 7, 4, 18, 3, 21, 1)
    assert (d.router_act, d.route_correction, d.route_renorm, d.route_on_input, d.act_kind) == (capi.ROUTER_SOFTMAX, 1, 0, 0, capi.ACT_SWISH)
    assert (descs[2].mlp_kind, descs[2].decay_rank, descs[2].decay_tau) == (capi.MLP_NONE, 1, 1.0)
    assert (descs[3].score_softcap, descs[3].rope_factor, descs[3].rope_dims, descs[3].route_identity, descs[3].shared_ff) == (0.0, 0.0, 8, 0, 0)


def test_bad_types_are_refused():
    cfg = arch_synth.tegolix_config(16, 8, [GL(1, 4, 4)], side_dim=3)
    cfg["layers"][0]["type"] = "retention"
    with pytest.raises(capi.PsCudaError):
        DESCRIBE(cfg, {})
    cfg = arch_synth.tegolix_config(16, 8, [GL(1, 4, 4, ff=8)], side_dim=3)
    cfg["layers"][0]["mlp"]["kind"] = "gated"
    with pytest.raises(capi.PsCudaError):
        DESCRIBE(cfg, {"l0.mix.a1": Shape(2, 16)})


def test_tensor_names_follow_the_layer_types():
    layers = [PA(2, 1, 4, 6, window=5, rwkv=(3, 2), ff=8, experts=3, top=2, identity=1, shared_ff=5), GL(2, 3, 5, ff=8), PA(1, 1, 4, 2, window=3, rwkv=(1, 4)), GL(1, 2, 3, ff=4, experts=2)]
    cfg = arch_synth.tegolix_config(16, 9, layers, side_dim=3)
    n = NAMES(cfg)
    t = arch_synth.tegolix_weights(cfg, seed=1, rank=7)
    used = {n["embed"], n["final_norm"], n["head"], n["token_embed"]}
    for ln in n["layers"]:
        for v in ln.values():
            used.update(v if isinstance(v, list) else [v])
        assert set(ln) <= set(capi.ARCH_LAYER_VECTORS_2) | {"norm", "q", "k", "v", "o", "router", "gate", "up", "down"}
    assert used == set(t)                                            # every stored tensor is named once, nothing else is
    assert t["side.embed"].shape == (9, 12) and t["l0.mlp.router"].shape == (4, 16) and t["l0.mix.right.u"].shape == (3, 2) and t["l1.mix.a1"].shape == (7, 16)
    assert "l2.norm2" not in t and "l2.ls2" not in t and "l2.side.gate" in t and "l3.mlp.shared.up" not in t


@pytest.mark.parametrize("dims,base,scaling", [(48, 10000.0, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}), (8, 100.0, YARN), (2, 50.0, None), (64, 5e5, {"factor": 1.5, "original": 4096, "fast": 8.0, "slow": 8.0})])
def test_rotation_table_of_the_backend(dims, base, scaling):
    import ctypes as C
    L = capi.load_library()
    out = (C.c_float * (dims // 2))()
    s = scaling or {"factor": 0.0, "original": 0, "fast": 0.0, "slow": 0.0}
    L.ps_cuda_host_rope_freq.restype = C.c_float
    L.ps_cuda_host_rope_freq.argtypes = [C.c_int, C.c_float, C.c_float, C.c_int, C.c_float, C.c_float, C.POINTER(C.c_float)]
    m = L.ps_cuda_host_rope_freq(dims, base, s["factor"], s["original"], s["fast"], s["slow"], out)
    f, want = R.yarn(dims, base, scaling)
    np.testing.assert_allclose(np.array(out[:]), f, rtol=2e-7)
    assert abs(m - want) < 1e-6


# ------------------------------------------------------------------------------------------------- the oracle by hand
def test_small_functions_by_hand():
    x, w = np.array([[1.0, 2.0, 3.0, 6.0]]), np.array([0.0, 1.0, -0.5, -2.0])
    np.testing.assert_allclose(R.offset_norm(x, w, 0.5), x / math.sqrt(50 / 4 + 0.5) * np.array([1.0, 2.0, 0.5, -1.0]))
    z = 0.7
    assert abs(float(R.gelu_tanh(np.array(z))) - 0.5 * z * (1 + math.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))) < 1e-15
    np.testing.assert_allclose(R.softcapped(np.array([0.0, 3.0, -1e9]), 2.0), [0.0, 2.0 * math.tanh(1.5), -2.0])
    assert R.softcapped(np.array([7.0]), None)[0] == 7.0


def test_window_edges():
    m = R.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5 and m[2].tolist() == [True] * 3 + [False] * 3


def test_rotated_values_depend_on_distance_only():
    """turning value j by j and the sum back by i leaves every weight's value turned by j - i: shifting all positions changes nothing"""
    rng = np.random.default_rng(0)
    v, f = rng.standard_normal((5, 6)), R.yarn(6, 40.0, None)[0]
    for shift in (0, 17):
        pos = np.arange(shift, shift + 5)[:, None]
        t = R.rotate_halves(v, pos * f)
        back = R.rotate_halves(np.tile(t[1], (5, 1)), -pos * f)[4]            # key 1 as query 4 sees it
        np.testing.assert_allclose(back, R.rotate_halves(v[1:2], np.array([[-3.0]]) * f)[0], atol=1e-12)
    a = 2.0
    np.testing.assert_allclose(R.rotate_halves(np.array([[1.0, 2.0, 5.0]]), np.array([[a]]), 1.5)[0], [1.5 * (math.cos(a) - 2 * math.sin(a)), 1.5 * (2 * math.cos(a) + math.sin(a)), 5.0])


def test_yarn_ramp_by_hand():
    f, m = R.yarn(8, 100.0, YARN)
    lo = max(math.floor(8 * math.log(40 / (2 * math.pi * 16)) / (2 * math.log(100))), 0)
    hi = min(math.ceil(8 * math.log(40 / (2 * math.pi * 2)) / (2 * math.log(100))), 7)
    for i in range(4):
        plain = 100.0 ** (-2 * i / 8)
        r = min(max((i - lo) / max(hi - lo, 0.001), 0), 1)
        assert abs(f[i] - (plain / 3 * r + plain * (1 - r))) < 1e-15
    assert abs(m - (0.1 * math.log(3) + 1)) < 1e-15


def test_recurrences_against_the_sum_over_the_past():
    rng = np.random.default_rng(1)
    T, d, dv = 6, 3, 4
    q, k, v, w, u = rng.standard_normal((T, d)), rng.standard_normal((T, d)), rng.standard_normal((T, dv)), rng.uniform(0.2, 1.0, (T, d)), rng.standard_normal(d)
    g, tm = R.gated_recurrence(q, k, v, w), R.time_mix_recurrence(q, k, v, w, u)
    for t in range(T):
        og, ot = np.zeros(dv), np.zeros(dv)
        for j in range(t + 1):
            og += (q[t] * np.prod(w[j + 1:t + 1], axis=0)) @ k[j] * v[j]
            ot += (q[t] * (u if j == t else np.prod(w[j + 1:t], axis=0))) @ k[j] * v[j]
        np.testing.assert_allclose(g[t], og, atol=1e-12)
        np.testing.assert_allclose(tm[t], ot, atol=1e-12)


def test_decay_root():
    cfg = arch_synth.tegolix_config(6, 5, [GL(1, 2, 2, tau=3.0)], side_dim=2)
    t = {k: np.asarray(v, np.float64) for k, v in arch_synth.tegolix_weights(cfg, seed=2).items()}
    z = np.array([-40.0, -1.0, 0.0, 2.0])
    np.testing.assert_allclose(np.exp(-R.softplus(-z) / 3.0), R.sigmoid(z) ** (1 / 3.0), rtol=1e-12)
    h = np.random.default_rng(3).standard_normal((4, 6))
    alpha = R.sigmoid((h @ t["l0.mix.a1"].T) @ t["l0.mix.a2"].T + t["l0.mix.a2.b"]) ** (1 / 3.0)
    o = R.gated_recurrence(h @ t["l0.mix.q"].T / math.sqrt(2), h @ t["l0.mix.k"].T, h @ t["l0.mix.v"].T, alpha)
    want = (o / np.sqrt((o * o).mean(-1, keepdims=True) + 1e-6) * t["l0.mix.norm"] * R.silu(h @ t["l0.mix.g"].T)) @ t["l0.mix.o"].T
    np.testing.assert_allclose(R.gla(h, cfg["layers"][0]["mixer"], t, "l0.mix.", 1e-6), want, atol=1e-12)


def test_routing_by_hand():
    z = np.log(np.array([[0.5, 0.3, 0.15, 0.05]]))
    np.testing.assert_allclose(R.route(z, np.zeros(4), 2), [[0.5, 0.3, 0, 0]])
    np.testing.assert_allclose(R.route(z, np.array([0, 0, 0.2, 0.0]), 2), [[0.5, 0, 0.15, 0]])     # the correction chooses, the score weighs
    np.testing.assert_allclose(R.route(z, np.array([-1.0, -1.0, -1.0, -0.1]), 1), [[0, 0, 0, 0.05]])


def test_identity_experts_pass_the_input_on():
    cfg = arch_synth.tegolix_config(6, 5, [GL(1, 2, 2, ff=3, experts=2, top=3, identity=2)], side_dim=2)
    t = {k: np.asarray(v, np.float64) for k, v in arch_synth.tegolix_weights(cfg, seed=4).items()}
    t["l0.mlp.correction"] = np.array([-9.0, 0.0, 0.0, 0.0])
    h = np.random.default_rng(5).standard_normal((3, 6))
    e = np.exp(h @ t["l0.mlp.router"].T)
    s = e / e.sum(-1, keepdims=True)
    np.testing.assert_allclose(R.mixture(h, cfg["layers"][0]["mlp"], t, "l0.mlp."), s[:, 1:2] * R.unit(h, t, "l0.mlp.e1.", R.silu) + (s[:, 2:3] + s[:, 3:4]) * h)


def test_layer_by_hand_and_causality():
    cfg = arch_synth.tegolix_config(12, 20, [PA(2, 1, 4, 6, window=3, rwkv=(2, 3), ff=8), GL(2, 3, 4)], side_dim=5)
    t = {k: np.asarray(v, np.float64) for k, v in arch_synth.tegolix_weights(cfg, seed=6).items()}
    toks = np.array([3, 1, 4, 1, 5, 9, 2])
    taps = []
    lg = R.forward(cfg, t, toks, taps)
    x, eps, l = t["embed"][toks], 1e-6, cfg["layers"][0]
    rms = lambda a: a / np.sqrt((a * a).mean(-1, keepdims=True) + eps)
    h = rms(x) * (1 + t["l0.norm1"])
    m = l["mixer"]
    y = m["left_scale"] * R.attention(h, m["left"], t, "l0.mix.left.", eps) + m["right_scale"] * R.time_mix(h, m["right"], t, "l0.mix.right.", eps)
    x = x + rms(y) * (1 + t["l0.norm1b"]) * t["l0.ls1"]
    h = rms(x) * (1 + t["l0.norm2"])
    y = (np.maximum(h @ t["l0.mlp.gate"].T, 0) * (h @ t["l0.mlp.up"].T)) @ t["l0.mlp.down"].T
    x = x + rms(y) * (1 + t["l0.norm2b"]) * t["l0.ls2"]
    y = (R.gelu_tanh(x @ t["l0.side.gate"].T) * t["side.embed"][toks][:, :5]) @ t["l0.side.proj"].T
    x = x + rms(y) * t["l0.side.norm"]
    np.testing.assert_allclose(taps[0], x, atol=1e-12)
    np.testing.assert_allclose(lg, rms(taps[1]) * (1 + t["final.norm"]) @ t["head"].T, atol=1e-12)
    np.testing.assert_allclose(R.forward(cfg, t, toks[:4]), lg[:4], atol=1e-10)      # a later position never changes an earlier one


def test_time_mix_reads_the_token_before():
    cfg = arch_synth.tegolix_config(8, 20, [PA(1, 1, 4, 4, window=3, rwkv=(2, 2))], side_dim=2)
    t = {k: np.asarray(v, np.float64) for k, v in arch_synth.tegolix_weights(cfg, seed=7).items()}
    m, p = cfg["layers"][0]["mixer"]["right"], "l0.mix.right."
    h = np.random.default_rng(8).standard_normal((3, 8))
    first = R.time_mix(h[:1], m, t, p, 1e-6)
    mix = lambda s: h[:1] * (1 - t[p + "mu." + s])                               # nothing stands before the first token
    r, k, v = (mix(s) @ t[p + s].T for s in "rkv")
    o = np.concatenate([((t[p + "u"][i] * k[0, 2 * i:2 * i + 2]) @ r[0, 2 * i:2 * i + 2]) * v[0, 2 * i:2 * i + 2] for i in range(2)]).reshape(2, 2)
    o = (o / np.sqrt((o * o).mean(-1, keepdims=True) + 1e-6)).reshape(1, 4)
    np.testing.assert_allclose(first, (o * t[p + "norm"] * R.silu(mix("g") @ t[p + "g"].T)) @ t[p + "o"].T, atol=1e-12)
    other = h.copy()
    other[1] += 1.0
    a, b = R.time_mix(h, m, t, p, 1e-6), R.time_mix(other, m, t, p, 1e-6)
    np.testing.assert_allclose(a[0], b[0])
    assert np.abs(a[2] - b[2]).max() > 1e-3


def test_configuration_survives_json():
    cfg = arch_synth.tegolix_config(16, 8, [PA(2, 1, 4, 4, window=9, rwkv=(1, 4), scaling=YARN)], side_dim=3)
    assert json.loads(json.dumps(cfg)) == cfg
