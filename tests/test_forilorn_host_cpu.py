"""Host-side tests of the Forilorn design: configuration, layer records, state, engine descriptors, synthetic models, and closed
forms of the oracle's own pieces.  No GPU."""

import math

import pytest
import torch

from dia_tts_prune_b200 import synthetic as SY
from dia_tts_prune_b200.lm_config import ForilornConfig, load_config
from oracle import forilorn_oracle as O

CFG = SY.forilorn_config(width=24, kinds=["attention", "latent_attention"], heads=4, kv_heads=2, dim=6, vocab=31, chunk=5, lat_heads=3,
                         lat_dim=8, rot_dim=4, lat_vdim=7, q_rank=9, kv_rank=10, window=3, ff=20, rot_dims=4, buckets=13, scale=2.5,
                         residual_mult=0.4)


def test_configuration_checks():
    cfg = load_config(CFG)
    assert isinstance(cfg, ForilornConfig) and cfg.layers[0].mixer.mask.size == 5 and cfg.embedding.bigram.buckets == 13
    cfg.check()

    def broken(i, **over):
        raw = {**CFG, "layers": [dict(lc) for lc in CFG["layers"]]}
        raw["layers"][i]["mixer"] = {**raw["layers"][i]["mixer"], **over}
        return load_config(raw)

    for i, over in ((0, {"kv_heads": 3}), (0, {"vdim": 7}), (0, {"rot": {"base": 10.0, "dims": 8}}), (0, {"rot": {"base": 10.0, "dims": 3}}),
                    (1, {"rot": {"base": 10.0, "dims": 6}})):
        with pytest.raises(ValueError):
            broken(i, **over).check()
    with pytest.raises(ValueError):
        broken(0, mask={"size": 0})
    with pytest.raises(ValueError):
        load_config({**CFG, "layers": [{"type": "retention", "mixer": {}}]})
    bare = load_config({**CFG, "embedding": {"scale": 1.0}, "layers": [{**CFG["layers"][0], "mlp": None}]})
    assert bare.embedding.bigram is None and bare.layers[0].mlp is None


def layers_and_state(**kw):
    from dia_tts_prune_b200.lm_model import build_forilorn_layers
    from dia_tts_prune_b200.lm_state import PagedState
    w = SY.forilorn_weights(CFG, 3)
    layers, final = build_forilorn_layers(ForilornConfig.model_validate(CFG), w, torch.device("cpu"))
    st = PagedState([ly.state_spec() for ly in layers], 24, 0, 40, torch.device("cpu"), page_size=4, max_sequences=3, **kw)
    return w, layers, final, st


def test_layer_records_stack_projections_and_add_one_to_norm_weights():
    w, layers, final, _ = layers_and_state()
    a, b = layers
    assert a.n_in == 24 + 12 + 24 and torch.equal(a.w_in[:24], w["l0.mix.q"]) and torch.equal(a.w_in[24:36], w["l0.mix.k"])
    assert torch.equal(a.w_in[36:], w["l0.mix.g"]) and a.mixer.chunk == 5 and a.mixer.window == 0 and not a.mixer.own_values
    assert a.mixer.q_norm is None and a.mixer.sink is None
    # query latent 9, latent 10 and turned part 4, one gate row per head: 26 rows, padded to 28
    assert b.n_in == 28 and torch.equal(b.w_in[:9], w["l1.mix.dq"]) and torch.equal(b.w_in[9:23], w["l1.mix.dkv"])
    assert torch.equal(b.w_in[23:26], w["l1.mix.g"]) and b.w_in[26:].abs().max() == 0
    assert b.mixer.window == 3 and b.mixer.head_gate and b.mixer.kv_rank == 10 and b.mixer.sink is None
    for ly, i in ((a, 0), (b, 1)):
        assert ly.norm1 is None and ly.norm2 is None and ly.ff.act == "gelu" and float(ly.hc1.w_out) == pytest.approx(0.4)
        assert torch.equal(ly.norm1_out.w, 1.0 + w[f"l{i}.norm1"].float()) and torch.equal(ly.norm2_out.w, 1.0 + w[f"l{i}.norm2"].float())
    assert torch.equal(final.w, 1.0 + w["final.norm"].float())


def test_state_keeps_tokens_on_the_page_table():
    _, layers, _, st = layers_and_state(keep_tokens=True)
    assert st.token_pages.shape == (13, 4) and st.token_pages.dtype == torch.int32
    assert st.record_state(0).k_pages.shape == (13, 2, 4, 6) and st.record_state(1).latent_pages.shape == (13, 4, 14)
    assert layers_and_state()[3].token_pages is None


def test_records_fill_the_engine_descriptors():
    from dia_tts_prune_b200 import _lm_lib as L
    from dia_tts_prune_b200.lm_layers import BigramEmbedding
    w, layers, _, st = layers_and_state(keep_tokens=True)
    recs = (L.Layer * 2)()
    for i, ly in enumerate(layers):
        ly.fill(recs[i], st.record_state(i))
    a, b = recs
    assert a.form == L.FORM_STREAMS and a.streams == 1 and a.mixer == L.MIXER_ROTARY_ATTENTION and a.values_are_keys == 1
    assert a.chunk == 5 and a.window == 0 and a.mixer_gate == L.GATE_SIGMOID and a.q_norm is None and a.sink is None
    assert a.norm_mix_in.w is None and a.norm_ff_in.w is None and a.norm_mix_out.kind == L.NORM_RMS
    assert a.norm_mix_out.w == layers[0].norm1_out.w.data_ptr() and a.norm_ff_out.w == layers[0].norm2_out.w.data_ptr()
    assert a.ff == L.FF_DENSE and a.act == L.ACT_GELU and a.dense_ff == 20
    assert b.mixer == L.MIXER_LATENT_ATTENTION and b.mixer_gate == L.GATE_SIGMOID_HEAD and b.window == 3 and b.chunk == 0
    assert (b.q_rank, b.kv_rank, b.rot_dim, b.rot_dims) == (9, 10, 4, 4)
    m = L.Model()
    big = BigramEmbedding(w["bigram"], buckets=13, mul_prev=13 * 10 ** 15 + 5, mul_cur=40, device=torch.device("cpu"))
    big.fill(m, st)
    assert (m.bigram_buckets, m.bigram_mul_prev, m.bigram_mul_cur) == (13, 5, 1) and m.token_pages == st.token_pages.data_ptr()


def test_stream_layers_without_input_norms_have_rules():
    from dia_tts_prune_b200.lm_layers import DenseUnit, HyperConnection, RmsNorm, StreamLayer
    _, layers, _, _ = layers_and_state()
    mixer, dev, one = layers[0].mixer, torch.device("cpu"), HyperConnection.residual(torch.device("cpu"))
    two = HyperConnection(torch.ones(2), torch.ones(2), torch.eye(2), dev)
    norm = RmsNorm(torch.ones(24), dev)
    for args, kw in (((None, two, mixer), {}), ((torch.ones(24), one, mixer), {"norm1_out": norm}), ((None, one, mixer), {"parallel": True})):
        with pytest.raises(ValueError):
            StreamLayer(*args, device=dev, **kw)
    with pytest.raises(ValueError):
        DenseUnit(torch.ones(4, 24), torch.ones(24, 4), act="silu")


def test_synthetic_models_have_the_oracles_tensors_and_the_registry_knows_the_design():
    from dia_tts_prune_b200.registry import architectures
    w, ref = SY.forilorn_weights(CFG, 5), O.random_weights(CFG, 5)
    assert {k: tuple(v.shape) for k, v in w.items()} == {k: tuple(v.shape) for k, v in ref.items()}
    assert torch.isfinite(O.forward(CFG, w, list(range(12)))).all()
    assert "forilorn" in architectures()


# ---- closed forms of the oracle's pieces ----------------------------------------------------------------------------------
def test_oracle_norm_and_gelu():
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    w = torch.tensor([0.0, 1.0], dtype=torch.float64)
    assert torch.allclose(O.zero_norm(x, w, 0.0), torch.tensor([[3.0, 8.0]], dtype=torch.float64) / math.sqrt(12.5))
    z = torch.tensor([-3.0, -1.0, 0.0, 0.5, 2.0], dtype=torch.float64)
    assert torch.allclose(O.gelu(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_oracle_pair_rows():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 4}
    assert O.bigram_rows([5, 7, 2], b) == [10, (15 + 28) % 10, (21 + 8) % 10]
    cfg = {"embedding": {"scale": 2.0, "bigram": b}}
    w = {"embed": torch.arange(8.0)[:, None], "bigram": 100.0 * torch.arange(11.0)[:, None]}
    assert O.embedding(cfg, w, [5, 7, 2]).flatten().tolist() == [1010.0, 314.0, 904.0]


def test_oracle_visibility():
    assert O.in_chunk(5, 4, 2) and not O.in_chunk(4, 3, 2) and not O.in_chunk(4, 5, 2) and O.in_chunk(4, 4, 1)
    assert O.in_window(5, 5, 1) and not O.in_window(5, 4, 1) and O.in_window(9, 5, 5) and not O.in_window(9, 4, 5)
    assert O.seen_mask(range(4), O.in_chunk, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 0, 1, 0], [0, 0, 1, 1]]


def test_oracle_rotation_turns_interleaved_pairs_and_keeps_the_mean_square():
    x = torch.randn(3, 2, 6, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    y = O.rotate(x, torch.tensor([0, 1, 7]), {"base": 100.0, "dims": 4})
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    c, s = math.cos(7 * 0.1), math.sin(7 * 0.1)                  # pair 1 turns by base^(-1/2) per position
    assert float(y[2, 1, 2]) == pytest.approx(float(x[2, 1, 2]) * c - float(x[2, 1, 3]) * s)
    assert float(y[2, 1, 3]) == pytest.approx(float(x[2, 1, 3]) * c + float(x[2, 1, 2]) * s)
    assert torch.allclose(O.rms_unit(y, 1e-3), O.rotate(O.rms_unit(x, 1e-3), torch.tensor([0, 1, 7]), {"base": 100.0, "dims": 4}))


def test_oracle_attention_of_lone_tokens_is_the_gated_raw_key():
    m = {"heads": 2, "kv_heads": 1, "dim": 3, "vdim": 3, "scale": 0.7, "mask": {"size": 1}}
    g = torch.Generator().manual_seed(1)
    p = {k: torch.randn(n, 5, generator=g, dtype=torch.float64) for k, n in (("q", 6), ("k", 3), ("g", 6))}
    p["o"] = torch.eye(6, dtype=torch.float64)
    h = torch.randn(4, 5, generator=g, dtype=torch.float64)
    k = (h @ p["k"].T).repeat(1, 2)
    assert torch.allclose(O.attention(h, p, m, 1e-6), k * torch.sigmoid(h @ p["g"].T))
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 2, "scale": 0.7, "mask": {"size": 1}, "rot": {"base": 9.0, "dims": 2}}
    p = {k: torch.randn(*s, generator=g, dtype=torch.float64) for k, s in (("dq", (3, 5)), ("dq.norm", (3,)), ("uq", (10, 3)), ("dkv", (6, 5)),
                                                                          ("dkv.norm", (4,)), ("uk", (6, 4)), ("uv", (4, 4)), ("g", (2, 5)))}
    p["o"] = torch.eye(4, dtype=torch.float64)
    c = O.rms_unit((h @ p["dkv"].T)[:, :4], 1e-6) * p["dkv.norm"]
    assert torch.allclose(O.latent_attention(h, p, m, 1e-6), (c @ p["uv"].T) * torch.sigmoid(h @ p["g"].T).repeat_interleave(2, dim=1))
