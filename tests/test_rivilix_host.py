"""Host side of the Rivilix decoder on CPU: configuration, weight packing, rotation table,
library parts, and the plain oracle's own consistency."""
import copy

import numpy as np
import pytest
import torch

import rivilix_oracle as R
from fastkernels_b200 import build
from fastkernels_b200.engine import DecodeEngine
from fastkernels_b200.models import registry
from fastkernels_b200.models.mixers import LatentAttention, Yarn, rope_table
from fastkernels_b200.models.rivilix import Rivilix, RivilixConfig
from fastkernels_b200.models.weights import DictSource, Packer


@pytest.mark.parametrize("name", sorted(R.MODELS))
def test_config_and_weights_of_a_folder(name, tmp_path):
    cfg = R.MODELS[name]
    w = R.random_weights(cfg, 3)
    R.write_folder(tmp_path, cfg, w)
    config, source = registry.load_folder(tmp_path, torch.float32)
    assert isinstance(config, RivilixConfig) and registry.model_class(config) is Rivilix
    assert config.order == R.order(cfg)
    assert {n: tuple(np.shape(a)) for n, a in w.items()} == config.tensor_shapes()
    for n, a in w.items():
        assert np.array_equal(source.get(n).float().numpy(), np.asarray(a, np.float32))
    parts = registry.library_parts(tmp_path)
    assert set(parts) <= set(build.COMPONENT_SOURCES) and "latent" in parts


def test_loop_positions():
    layers = [R.memory_layer() for _ in range(4)]
    for loop, want in (((0, 4, 2), [0, 1, 2, 3, 0, 1, 2, 3]), ((1, 3, 2), [0, 1, 2, 1, 2, 3]),
                       (None, [0, 1, 2, 3]), ((2, 3, 1), [0, 1, 2, 3])):
        config = registry._module("Rivilix").config_from_json(
            R.model_config(layers, loop=loop), DictSource({}))
        assert [i for i, _ in config.order] == want
        begins = [k for k, (_, b) in enumerate(config.order) if b]
        assert len(begins) == (loop[2] if loop else 0)
        assert all(want[k] == loop[0] for k in begins)
    with pytest.raises(ValueError, match="loop"):
        registry._module("Rivilix").config_from_json(R.model_config(layers, loop=(2, 5, 2)),
                                                     DictSource({}))


@pytest.mark.parametrize("change,text", [(dict(type="other"), "unknown mixer"),
                                         (dict(mlp={"kind": "sparse"}), "unknown feed")])
def test_unknown_branches_are_refused(change, text):
    cfg = R.model_config([{**R.latent_layer(), **change}])
    with pytest.raises(ValueError, match=text):
        registry._module("Rivilix").config_from_json(cfg, DictSource({}))
    cfg = R.model_config([R.latent_layer()])
    cfg["layers"][0]["mixer"]["rot"]["dims"] = 4
    with pytest.raises(ValueError, match="rotated"):
        registry._module("Rivilix").config_from_json(cfg, DictSource({}))


@pytest.mark.parametrize("dims,base,yarn", [(8, 900.0, (4.0, 60, 8.0, 0.5)),
                                            (64, 1e4, (40.0, 4096, 32.0, 1.0)),
                                            (10, 5e5, (16.0, 300, 2.0, 1.9)),
                                            (2, 100.0, (2.0, 8192, 32.0, 1.0)), (12, 300.0, None)])
def test_rotation_table(dims, base, yarn):
    scaling = Yarn(*yarn) if yarn else None
    t = rope_table(900, dims, base, "cpu", scaling).double().numpy()
    f, mscale = R.rotary_frequencies(dims, base, dict(zip(
        ("factor", "original", "fast", "slow"), yarn)) if yarn else None)
    p = np.arange(900)[:, None]
    np.testing.assert_allclose(t[:, :dims // 2], np.cos(p * f) * mscale, atol=3e-7)
    np.testing.assert_allclose(t[:, dims // 2:], np.sin(p * f) * mscale, atol=3e-7)


@pytest.mark.parametrize("sizes", [(5, 24, 8, 20, 40), (1, 40, 40, 8, 16), (3, 15, 10, 33, 23),
                                   (2, 120, 40, 136, 200)])
def test_packed_weights_of_latent_attention(sizes):
    """Absorbed and expanded products on the cached row equal keys, values and output of the
    plain ones; padding may hold anything finite."""
    h, dim, rot, vdim, rank = sizes
    rs = np.random.RandomState(sum(sizes))
    width = 24
    tensors = {"m.q": rs.randn(h * (dim + rot), width), "m.dkv": rs.randn(rank + rot, width),
               "m.dkv.norm": rs.rand(rank), "m.uk": rs.randn(h * dim, rank),
               "m.uv": rs.randn(h * vdim, rank), "m.o": rs.randn(width, h * vdim)}
    att = LatentAttention(h, dim, rot, vdim, rank, 1.0, 10.0, None, 0, 1e-5, torch.bfloat16)
    att.dtype = torch.float32
    w = Packer(DictSource({n: torch.from_numpy(a) for n, a in tensors.items()}), "cpu",
               torch.float32, width, 64)
    rows = att.load(w, "m.")
    assert {n: m.shape[0] for n, m in rows.items()} == att.sections
    x = torch.from_numpy(rs.randn(width)).float()
    q = (rows["q"] @ x).view(h, att.q_pitch)
    want_q = (torch.from_numpy(tensors["m.q"]).float() @ x).view(h, dim + rot)
    torch.testing.assert_close(q[:, :dim + rot], want_q)
    c = torch.from_numpy(rs.randn(rank)).float()
    key = (torch.from_numpy(tensors["m.uk"]).float() @ c).view(h, dim)
    value = (torch.from_numpy(tensors["m.uv"]).float() @ c).view(h, vdim)
    # the product reads the columns behind the unrotated part: they meet zero weights
    tail = torch.cat([(rows["q"] @ x), torch.full((16,), 5.0)])
    kd = att.w_key.shape[2]
    absorbed = torch.stack([att.w_key[i] @ tail[i * att.q_pitch:i * att.q_pitch + kd]
                            for i in range(h)])
    torch.testing.assert_close(absorbed @ c, (want_q[:, :dim] * key).sum(1), rtol=1e-4, atol=1e-3)
    lo = att.w_value.shape[2]
    cached = torch.cat([c, torch.full((lo,), 2.0)])[:lo]
    out = att.w_value @ cached
    torch.testing.assert_close(out[:, :vdim], value, rtol=1e-4, atol=1e-3)
    packed = att.pack_output(torch.from_numpy(tensors["m.o"]).float())
    full = torch.zeros(att.out_columns)
    full[:h * att.v_pitch] = out.reshape(-1)
    torch.testing.assert_close(packed @ full, torch.from_numpy(tensors["m.o"]).float() @
                               value.reshape(-1), rtol=1e-4, atol=1e-2)
    assert att.expandable == (dim + rot <= 128 and vdim <= 128)
    if att.expandable:
        row = torch.zeros(att.row)
        row[:rank], row[rank:rank + rot] = c, torch.arange(rot) + 1.0
        kv = (att.w_expand @ row).view(2, h, 128)
        torch.testing.assert_close(kv[0, :, :dim], key, rtol=1e-4, atol=1e-3)
        assert torch.equal(kv[0, :, dim:dim + rot], (torch.arange(rot) + 1.0).expand(h, rot))
        torch.testing.assert_close(kv[1, :, :vdim], value, rtol=1e-4, atol=1e-3)
        assert torch.count_nonzero(kv[0, :, dim + rot:]) == 0
        assert torch.count_nonzero(kv[1, :, vdim:]) == 0


def test_engine_pools_states_and_release(tmp_path):
    """One pool per pass of an attention layer, one state per pass of a memory; what a
    sequence holds comes back."""
    cfg = R.MODELS["loop"]
    R.write_folder(tmp_path, cfg, R.random_weights(cfg, 1))
    config, source = registry.load_folder(tmp_path, torch.float32)
    eng = DecodeEngine(config, max_num_seqs=2, max_model_len=200, num_kv_blocks=7, device="cpu",
                       init_scale=None)
    eng.load_weights(source)
    assert [b.chunk for b in eng.span_blocks] == [None]
    first, att, last = (layer.mixer for layer in eng.model.layers)
    assert len(att.caches) == 3 and len(first.states) == 3 and len(last.states) == 1
    assert att.caches[0].shape == (7, 64, 1, 64)
    assert first.states[0][0].shape == (2, 2, 9, 8) and first.states[0][1].shape == (2, 2, 12)
    assert eng.model.last_ids.shape == (2,)
    a = eng.open_sequence()
    eng.span_blocks[0].extend(a, 0, 130)
    eng.finish(a)
    assert len(eng.span_blocks[0].free) == 7 and len(eng.state_slots.free) == 2
    for i, k in ((0, None), (1, 3)):
        assert eng.model.runs[i] == (i, 0, i == 0)
    assert [r[1] for r in eng.model.runs] == [0, 0, 1, 1, 2, 2, 0]


# ------------------------------------------------------------------------- the oracle
def test_oracle_memory_in_two_pieces_and_against_sums():
    """Split in two it gives what it gives in one piece; and the stabilized recurrence
    equals the weighted sums it stands for."""
    rs = np.random.RandomState(0)
    t, h, d, e = 9, 2, 5, 3
    q, k, v = rs.randn(t, h, d), rs.randn(t, h, d), rs.randn(t, h, e)
    i, f = R.mlstm_gates(rs.randn(t, h) * 4, rs.randn(t, h) * 4 + 2, 6.0)
    o, s = R.mlstm_memory(q, k, v, i, f)
    o1, s1 = R.mlstm_memory(q[:4], k[:4], v[:4], i[:4], f[:4])
    o2, s2 = R.mlstm_memory(q[4:], k[4:], v[4:], i[4:], f[4:], s1)
    np.testing.assert_allclose(np.concatenate([o1, o2]), o)
    for a, b in zip(s, s2):
        np.testing.assert_allclose(a, b)
    for a in range(t):
        for g in range(h):
            wt = [np.exp(f[b + 1:a + 1, g].sum() + i[b, g]) for b in range(a + 1)]
            num = sum(x * (q[a, g] @ k[b, g]) * v[b, g] for b, x in enumerate(wt))
            den = sum(x * (q[a, g] @ k[b, g]) for b, x in enumerate(wt))
            m = max([f[:a + 1, g].sum()] + [np.log(x) for x in wt])
            want = num * np.exp(-m) / (max(abs(den) * np.exp(-m), np.exp(-m)) + 1e-6)
            np.testing.assert_allclose(o[a, g], want, rtol=1e-9)


def test_oracle_bigram_rows():
    assert R.bigram_rows([4, 0, 6], 37, 11, 5).tolist() == [37, 44 % 37, 30]
    assert R.bigram_rows([4], 1, 2, 3).tolist() == [1]


def rel(got, want):
    return (np.sqrt(np.mean((got - want) ** 2, axis=1)) / np.sqrt(np.mean(want ** 2))).max()


@pytest.mark.parametrize("name", sorted(R.MODELS))
def test_mistakes_show_in_the_logits(name):
    """The random models of the GPU tests are sharp enough: a lost state or cache, a missing
    previous token, one expert fewer or a plain rotation moves some position by far more
    than the tolerance there in fp32."""
    cfg = R.MODELS[name]
    w = R.random_weights(cfg, len(name))
    s = np.random.RandomState(11).randint(0, cfg["vocab"], size=140)
    want = R.forward(s, w, cfg)
    assert rel(R.forward(s[70:], w, cfg)[:20], want[70:90]) > 0.3
    if cfg.get("embedding"):
        c = copy.deepcopy(cfg)
        c["embedding"]["bigram"]["mul_prev"] += 1
        if c["embedding"]["bigram"]["buckets"] > 1:
            assert rel(R.forward(s, w, c), want) > 0.3
    for i, layer in enumerate(cfg["layers"]):
        c = copy.deepcopy(cfg)
        m = c["layers"][i]["mixer"]
        if layer["type"] == "latent_attention":
            if "scaling" in m["rot"] and m["rot_dim"] > 2 and m["rot"]["scaling"]["factor"] > 1:
                del m["rot"]["scaling"]
                assert rel(R.forward(s, w, c), want) > 0.15
        else:
            m["gate_cap"] *= 0.2
            assert rel(R.forward(s, w, c), want) > 0.15
        f = c["layers"][i].get("mlp") or {}
        if f.get("kind") == "moe" and f["router"]["top"] > 1:
            c = copy.deepcopy(cfg)
            c["layers"][i]["mlp"]["router"]["top"] -= 1
            assert rel(R.forward(s, w, c), want) > 0.03
