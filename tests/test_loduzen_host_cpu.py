"""Host-side tests of the Loduzen design: configuration, layer records, state specs, synthetic models, and closed forms of the
oracle's own pieces.  No GPU."""

import math

import pytest
import torch

from dia_tts_prune_b200 import synthetic as SY
from dia_tts_prune_b200.lm_config import LoduzenConfig, load_config
from oracle import loduzen_oracle as O

CFG = SY.loduzen_config(width=24, kinds=["parallel", "mamba2"], heads=3, kv_heads=1, dim=6, vocab=31, window=5, lin_heads=2, lin_dim=5,
                        lin_vdim=7, ssm_heads=4, ssm_vdim=3, ssm_state=10, ssm_groups=2, norm_groups=2, taps=3, ff=9, side=4, rot_dims=4,
                        yarn={"factor": 2.0, "original": 50, "fast": 4.0, "slow": 1.0})


def test_configuration_checks():
    cfg = load_config(CFG)
    assert isinstance(cfg, LoduzenConfig) and cfg.layers[0].mixer.left.mask.size == 5 and cfg.token_side.dim == 4
    cfg.check()

    def broken(layer, **over):
        raw = {**CFG, "layers": [dict(lc) for lc in CFG["layers"]]}
        m = dict(raw["layers"][layer]["mixer"])
        if layer == 0:
            m["left"] = {**m["left"], **over}
        else:
            m.update(over)
        raw["layers"][layer]["mixer"] = m
        return load_config(raw)

    for layer, over in ((0, {"kv_heads": 2}), (0, {"vdim": 8}), (0, {"rot": {"base": 10.0, "dims": 8}}), (0, {"rot": {"base": 10.0, "dims": 3}}),
                        (1, {"groups": 3}), (1, {"norm_groups": 5})):
        with pytest.raises(ValueError):
            broken(layer, **over).check()
    with pytest.raises(ValueError):
        load_config({**CFG, "layers": [{"type": "convolution", "mixer": {}}]})
    bare = load_config({**CFG, "token_side": None, "layers": [{**CFG["layers"][0], "mlp": None}]})
    assert bare.token_side is None and bare.layers[0].mlp is None


def test_layer_records_stack_both_mixers_and_share_the_token_table():
    from dia_tts_prune_b200.lm_model import build_loduzen_layers
    cfg, dev = LoduzenConfig.model_validate(CFG), torch.device("cpu")
    w = SY.loduzen_weights(CFG, 3, rank=5)
    layers, final = build_loduzen_layers(cfg, w, dev)
    left, right = layers[0].mixer.parts
    # left: 18 + 6 rows; right: 10 + 10 + 14 + 14 + 5 = 53 rows, padded to 56
    assert layers[0].n_in == 24 + 56 and layers[0].mixer.part_rows == [24, 56] and layers[0].w_o.shape == (24, 18 + 14)
    assert torch.equal(layers[0].w_in[:18], w["l0.mix.left.q"]) and torch.equal(layers[0].w_in[18:24], w["l0.mix.left.k"])
    assert torch.equal(layers[0].w_in[24:34], w["l0.mix.right.q"]) and torch.equal(layers[0].w_in[24 + 48:24 + 53], w["l0.mix.right.a1"])
    assert layers[0].w_in[77:].abs().max() == 0
    assert torch.equal(layers[0].w_o[:, :18], w["l0.mix.left.o"]) and torch.equal(layers[0].w_o[:, 18:], w["l0.mix.right.o"])
    assert left.window == 5 and not left.own_values and left.sink.abs().max() == 0 and right.rank == 5
    assert layers[1].n_in == 12 * 2 + 2 * 2 * 10 + 4 and layers[1].mixer.channels == 12 + 40
    assert layers[0].side.table is layers[1].side.table and [ly.side.offset for ly in layers] == [0, 4]
    assert layers[0].ff.act == "gelu" and layers[0].rms and not layers[0].parallel


def test_state_of_a_pair_has_a_record_per_part():
    from dia_tts_prune_b200.lm_model import build_loduzen_layers
    from dia_tts_prune_b200.lm_state import PagedState
    layers, _ = build_loduzen_layers(LoduzenConfig.model_validate(CFG), SY.loduzen_weights(CFG, 3), torch.device("cpu"))
    st = PagedState([ly.state_spec() for ly in layers], 24, 0, 40, torch.device("cpu"), page_size=4, max_sequences=3)
    pair, ssm = st.record_state(0), st.record_state(1)
    assert pair.k_pages is None and pair.rec_state is None and len(pair.parts) == 2
    assert pair.parts[0].k_pages.shape == pair.parts[0].v_pages.shape == (13, 1, 4, 6)
    assert pair.parts[1].rec_state.shape == (3, 2, 7, 5) and pair.parts[1].k_pages is None
    assert ssm.rec_state.shape == (3, 4, 3, 10) and ssm.conv_tail.shape == (3, 2, 52) and ssm.parts == ()
    seq = st.open("a")
    st.reserve(seq, 9)
    assert len(seq.pages) == 3
    st.close("a")
    assert st.free_pages == 13


def test_records_fill_the_engine_descriptors():
    import ctypes as C
    from dia_tts_prune_b200 import _lm_lib as L
    from dia_tts_prune_b200.lm_model import build_loduzen_layers
    from dia_tts_prune_b200.lm_state import PagedState
    layers, _ = build_loduzen_layers(LoduzenConfig.model_validate(CFG), SY.loduzen_weights(CFG, 3), torch.device("cpu"))
    st = PagedState([ly.state_spec() for ly in layers], 24, 0, 40, torch.device("cpu"), page_size=4, max_sequences=3)
    recs = (L.Layer * 2)()
    for i, ly in enumerate(layers):
        ly.fill(recs[i], st.record_state(i))
    a = recs[0]
    assert a.mixer == L.MIXER_PAIR and a.form == L.FORM_STREAMS and a.streams == 1 and a.act == L.ACT_GELU_GLU and a.dense_ff == 9
    left, right = (C.cast(a.part[q], C.POINTER(L.Layer)).contents for q in range(2))
    assert left.mixer == L.MIXER_ROTARY_ATTENTION and left.values_are_keys == 1 and left.window == 5 and left.n_in == 24
    assert abs(left.rot_amp - (0.1 * math.log(2.0) + 1.0)) < 1e-6 and left.rot_dims == 4 and left.mixer_gate == L.GATE_NONE
    assert right.mixer == L.MIXER_GATED_LINEAR and right.decay_tau == 16.0 and right.rec_state == st.record_state(0).parts[1].rec_state.data_ptr()
    assert abs(a.part_scale[0] - 0.8) < 1e-6 and abs(a.part_scale[1] - 0.6) < 1e-6
    b = recs[1]
    assert b.mixer == L.MIXER_MAMBA2 and (b.dim, b.kv_heads, b.vdim, b.conv_taps, b.norm_groups) == (10, 2, 3, 3, 2)
    assert b.side_dim == 4 and b.side_off == 4 and b.side_ld == 8 and b.side_table == a.side_table


def test_yarn_angles_against_hand_made_numbers():
    from types import SimpleNamespace
    from dia_tts_prune_b200.lm_layers import rotary_angles, yarn_angles
    plain, amp = yarn_angles(100.0, 8)
    assert amp == 1.0 and torch.equal(plain, rotary_angles(100.0, 8))
    # base e^2, 8 channels: the pair that makes t turns in 2 pi e^2 t0 positions is 8 ln(e^2 t0 / t) / 4 = 2 (2 + ln t0 - ln t)
    sc = SimpleNamespace(factor=5.0, original=2.0 * math.pi * math.e ** 2, fast=math.e ** 1.4, slow=math.e ** 0.4)
    got, amp = yarn_angles(math.e ** 2, 8, sc)                   # the ramp runs from floor(1.2) = 1 to ceil(3.2) = 4
    want = []
    for i in range(4):
        f, r = math.e ** (-0.5 * i), min(max((i - 1) / 3.0, 0.0), 1.0)
        want.append(f / 5.0 * r + f * (1.0 - r))
    assert torch.allclose(got, torch.tensor(want), rtol=1e-6) and abs(amp - (1.0 + 0.1 * math.log(5.0))) < 1e-12
    oracle, oamp = O.frequencies({"base": math.e ** 2, "dims": 8, "scaling": vars(sc)})
    assert torch.allclose(got, torch.tensor(oracle, dtype=torch.float32), rtol=1e-6) and oamp == amp


def test_synthetic_models_have_the_oracles_tensors():
    w, ref = SY.loduzen_weights(CFG, 5, rank=12), O.random_weights(CFG, 5, rank=12)
    assert {k: tuple(v.shape) for k, v in w.items()} == {k: tuple(v.shape) for k, v in ref.items()}
    assert torch.isfinite(O.forward(CFG, w, list(range(12)))).all()


# ---- closed forms of the oracle's pieces ----------------------------------------------------------------------------------
def test_oracle_gelu_softplus_and_convolution():
    z = torch.tensor([-3.0, -1.0, 0.0, 0.5, 2.0], dtype=torch.float64)
    assert torch.allclose(O.gelu(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)
    assert torch.allclose(O.softplus(z), torch.log(1 + torch.exp(z)), atol=1e-12) and float(O.softplus(torch.tensor(800.0))) == 800.0
    u, w = torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[2.0, 3.0]])
    assert O.causal_conv(u, w, torch.tensor([0.5])).flatten().tolist() == [3.5, 32.5, 320.5]


def test_oracle_window_of_one_is_a_sigmoid_of_the_own_score():
    m = {"heads": 2, "kv_heads": 1, "dim": 3, "vdim": 3, "scale": 0.7, "mask": {"size": 1}}
    g = torch.Generator().manual_seed(1)
    p = {k: torch.randn(n, 5, generator=g, dtype=torch.float64) for k, n in (("q", 6), ("k", 3))}
    p.update({"q.norm": torch.ones(3, dtype=torch.float64), "k.norm": torch.full((3,), 2.0, dtype=torch.float64), "o": torch.eye(6, dtype=torch.float64)})
    h = torch.randn(4, 5, generator=g, dtype=torch.float64)
    got = O.window_attention(h, p, m, 0.0)
    q, k = (h @ p["q"].T).reshape(4, 2, 3), h @ p["k"].T
    s = (O.rms_unit(q, 0.0) * (2.0 * O.rms_unit(k, 0.0))[:, None]).sum(-1) * 0.7
    assert torch.allclose(got, (torch.sigmoid(s)[..., None] * k[:, None]).reshape(4, 6), atol=1e-12)


def test_oracle_recurrences_as_plain_double_sums():
    T, eps, g = 7, 0.0, torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)            # noqa: E731
    h = rnd(T, 4)
    m = {"heads": 1, "dim": 3, "vdim": 2, "tau": 4.0}
    p = {"q": rnd(3, 4), "k": rnd(3, 4), "v": rnd(2, 4), "g": rnd(2, 4), "a1": rnd(2, 4), "a2": rnd(3, 2), "a2.b": rnd(3),
         "norm": torch.ones(2, dtype=torch.float64), "o": torch.eye(2, dtype=torch.float64)}
    alpha = torch.sigmoid((h @ p["a1"].T) @ p["a2"].T + p["a2.b"]) ** 0.25
    q, k, v = h @ p["q"].T / math.sqrt(3.0), h @ p["k"].T, h @ p["v"].T
    o = torch.stack([sum((q[t] * k[s] * alpha[s + 1:t + 1].prod(dim=0)).sum() * v[s] for s in range(t + 1)) for t in range(T)])
    assert torch.allclose(O.gated_linear_attention(h, p, m, eps), O.rms_unit(o, 0.0) * O.silu(h @ p["g"].T), atol=1e-10)
    m = {"heads": 1, "vdim": 2, "state": 3, "groups": 1, "conv": 1, "norm_groups": 1}
    p = {"in": rnd(2 + 2 + 6 + 1, 4), "conv": torch.ones(8, 1, dtype=torch.float64), "conv.b": rnd(8), "dt_bias": rnd(1), "A_log": rnd(1),
         "D": rnd(1), "norm": torch.ones(2, dtype=torch.float64), "o": torch.eye(2, dtype=torch.float64)}
    pr = h @ p["in"].T
    xbc, dt = O.silu(pr[:, 2:10] + p["conv.b"]), torch.log1p(torch.exp(pr[:, 10] + p["dt_bias"]))
    x, B, C, a = xbc[:, :2], xbc[:, 2:5], xbc[:, 5:], torch.exp(-torch.exp(p["A_log"]) * dt)
    y = torch.stack([sum(dt[s] * a[s + 1:t + 1].prod() * (C[t] @ B[s]) * x[s] for s in range(t + 1)) + p["D"] * x[t] for t in range(T)])
    assert torch.allclose(O.mamba2(h, p, m, eps), O.rms_unit(y * O.silu(pr[:, :2]), 0.0), atol=1e-10)


def test_oracle_token_input_and_visibility():
    assert O.visible(5, 5, 1) and not O.visible(5, 4, 1) and not O.visible(4, 5, None) and O.visible(90, 0, None) and O.visible(9, 5, 5)
    p = {"gate": torch.tensor([[1.0, 0.0]]), "proj": torch.tensor([[3.0], [4.0]]), "norm": torch.tensor([1.0, 2.0])}
    got = O.token_input(torch.tensor([[2.0, 9.0]]), torch.tensor([[-1.0]]), p, 0.0)     # (3, 4) / rms = (3, 4) / sqrt(12.5), sign of e
    assert torch.allclose(got, torch.tensor([[-3.0, -8.0]]) / math.sqrt(12.5), atol=1e-6)
