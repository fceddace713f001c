"""Host side of the Pinuvik decoder on CPU: configuration, weight packing, page tables
of chunked spans, state slots, the trace runner's protocol, and the plain oracle's own
consistency."""
import io
import json
import struct

import numpy as np
import pytest
import torch

import pinuvik_oracle as P
from fastkernels_b200 import trace
from fastkernels_b200.cache import BlockManager, Sequence, StateSlots
from fastkernels_b200.engine import DecodeEngine
from fastkernels_b200.models import registry
from fastkernels_b200.models.mixers import RotaryAttention, rope_table
from fastkernels_b200.models.pinuvik import Pinuvik, PinuvikConfig
from fastkernels_b200.models.weights import DictSource, SafetensorsSource


def small(tmp_path, **kw):
    cfg = P.model_config([P.layer_config(), P.layer_config(chunk=40, ff=None, heads=3,
                                                           kv_heads=1, dim=20, rot=(8, 500.0))],
                         width=40, vocab=51, loop=(1, 2, 3), **kw)
    w = P.random_weights(cfg, 3, rank=6)
    P.write_folder(tmp_path, cfg, w)
    return cfg, w


def test_config_and_weights_of_a_folder(tmp_path):
    cfg, w = small(tmp_path)
    config, source = registry.load_folder(tmp_path, torch.float32)
    assert isinstance(config, PinuvikConfig) and registry.model_class(config) is Pinuvik
    assert config.order == [0, 1, 1, 1] == P.layer_order(cfg)
    assert [c.decay_rank for c in config.layers] == [6, 6]
    assert [c.chunk for c in config.layers] == [24, 40]
    assert config.layers[1].ff is None and config.layers[1].kv_heads == 1
    assert {n: tuple(np.shape(a)) for n, a in w.items()} == config.tensor_shapes()
    for name, a in w.items():
        assert tuple(source.shape(name)) == np.shape(a)
        assert np.array_equal(source.get(name).float().numpy(), np.asarray(a, np.float32))
    with pytest.raises(KeyError, match="l9"):
        source.get("l9.norm1")


def test_loop_positions():
    layers = [P.layer_config() for _ in range(4)]
    for loop, want in (((0, 4, 2), [0, 1, 2, 3, 0, 1, 2, 3]), ((1, 3, 2), [0, 1, 2, 1, 2, 3]),
                       (None, [0, 1, 2, 3]), ((2, 3, 1), [0, 1, 2, 3])):
        cfg = P.model_config(layers, loop=loop)
        assert P.layer_order(cfg) == want
        src = DictSource({f"l{i}.mix.right.w1": torch.zeros(5, 8) for i in range(4)})
        module = registry._module("Pinuvik")
        assert module.config_from_json(cfg, src).order == want


@pytest.mark.parametrize("change", [dict(type="other"), dict(mlp={"kind": "sparse", "ff": 8})])
def test_unknown_branches_are_refused(change):
    cfg = P.model_config([{**P.layer_config(), **change}])
    src = DictSource({"l0.mix.right.w1": torch.zeros(5, 8)})
    with pytest.raises(ValueError, match="unknown"):
        registry._module("Pinuvik").config_from_json(cfg, src)
    with pytest.raises(ValueError, match="unknown architecture"):
        registry._module("Nothing")


def test_llama_folder_goes_through_the_same_registry(tmp_path):
    from fastkernels_b200.candidate.L4.llama import LlamaConfig
    cfg = dict(architectures=["Qwen3ForCausalLM"], hidden_size=128, intermediate_size=256,
               num_hidden_layers=1, num_attention_heads=2, num_key_value_heads=1, head_dim=128,
               vocab_size=96, max_position_embeddings=256, rms_norm_eps=1e-6, rope_theta=1e6)
    rs = np.random.RandomState(0)
    a, m = "model.layers.0.self_attn.", "model.layers.0.mlp."
    shapes = {"model.embed_tokens.weight": (96, 128), "lm_head.weight": (96, 128),
              "model.norm.weight": (128,), a + "q_proj.weight": (256, 128),
              a + "k_proj.weight": (128, 128), a + "v_proj.weight": (128, 128),
              a + "o_proj.weight": (128, 256), a + "q_norm.weight": (128,),
              a + "k_norm.weight": (128,), m + "gate_proj.weight": (256, 128),
              m + "up_proj.weight": (256, 128), m + "down_proj.weight": (128, 256),
              "model.layers.0.input_layernorm.weight": (128,),
              "model.layers.0.post_attention_layernorm.weight": (128,)}
    w = {n: P.bf16(rs.randn(*s)) for n, s in shapes.items()}
    P.write_folder(tmp_path, cfg, w)
    config, source = registry.load_folder(tmp_path)
    assert isinstance(config, LlamaConfig) and config.qk_norm
    eng = DecodeEngine(config, max_num_seqs=2, max_model_len=128, num_kv_blocks=2, device="cpu",
                       init_scale=None)
    eng.load_weights(source)
    att = eng.model.model.layers[0].self_attn
    got = att.qkv_proj.weight.detach().float().numpy()
    assert np.array_equal(got[256:384], w[a + "k_proj.weight"].astype(np.float32))
    gu = eng.model.model.layers[0].mlp.gate_up_proj.weight.detach().float().numpy()
    assert np.array_equal(gu[256:], w[m + "up_proj.weight"].astype(np.float32))


def test_rope_table():
    t = rope_table(700, 12, 300.0, "cpu").numpy()
    for p in (0, 1, 13, 699):
        for i in range(6):
            ang = p * 300.0 ** (-2 * i / 12)
            assert abs(t[p, i] - np.cos(ang)) < 1e-6 and abs(t[p, 6 + i] - np.sin(ang)) < 1e-6
    assert rope_table(5, 0, 1.0, "cpu").shape == (5, 1)


@pytest.mark.parametrize("heads,kv,dim,dtype", [(6, 2, 40, torch.bfloat16), (5, 1, 128, torch.bfloat16),
                                                (6, 3, 30, torch.float32), (2, 2, 160, torch.bfloat16)])
def test_output_weight_follows_the_padding_of_heads(heads, kv, dim, dtype):
    att = RotaryAttention(heads, kv, dim, 1.0, 4, 10.0, 0, 1e-5, dtype)
    w = torch.randn(7, heads * dim)
    packed = att.pack_output(w)
    assert packed.shape[1] == att.out_columns and att.out_columns % 64 == 0
    x = torch.randn(heads, dim)
    xp = torch.full((kv, att.group, att.padded_dim), 3.0)     # pads must not matter
    for h in range(heads):
        xp[h // (heads // kv), h % (heads // kv), :dim] = x[h]
    xp = torch.nn.functional.pad(xp.reshape(-1), (0, att.out_columns - xp.numel()))
    torch.testing.assert_close(packed @ xp, w @ x.reshape(-1))
    if att.tensor_cores:
        assert att.padded_dim == 128 and att.group & (att.group - 1) == 0


def brute_slots(bm, seq, a, n):
    """Where extend must put each token, from first principles."""
    out = []
    for p in range(a, a + n):
        off = p if bm.chunk is None else p % bm.chunk
        out.append((off // bm.block_size, off % bm.block_size))
    return out


@pytest.mark.parametrize("chunk", [None, 10, 64, 7, 16])
def test_span_pages_in_portions(chunk):
    """Random portions: every segment sees exactly the keys of its chunk, at the page
    and offset they were written to; nothing is shared, everything comes back."""
    rs = np.random.RandomState(5)
    bm = BlockManager(200, 8, 0, chunk)
    seqs = [Sequence(i, 0) for i in range(3)]
    written = [dict() for _ in seqs]                       # position -> slot
    for _ in range(60):
        i = rs.randint(3)
        s, n = seqs[i], int(rs.choice([1, 2, 3, 9, 25]))
        a = s.num_tokens
        if a + n > 150:
            continue
        if n == 1 and a > 0:                               # as a decode step does
            s.num_tokens += 1
            bm.maybe_append_page(s)
            assert bm.pages_missing(s) == 0 and not bm.maybe_append_page(s)
            written[i][a] = bm.slot(s, a)
            segs = [(1, a - bm.base(a) + 1, np.array(s.table(0)))]
        else:
            segs, slots = bm.extend(s, a, n)
            s.num_tokens += n
            for p, sl in zip(range(a, a + n), slots):
                written[i][p] = int(sl)
            live = [x for t in seqs for x in t.table(0)] + bm._retired + bm.free
            assert len(live) == len(set(live)) == 200
            bm.flush()
        at = a
        for q_len, k_len, pages in segs:
            last = at + q_len - 1
            base = 0 if chunk is None else last // chunk * chunk
            assert k_len == last - base + 1
            for p in range(base, last + 1):
                off = p - base
                assert written[i][p] == pages[off // 8] * 8 + off % 8
            at += q_len
        # only the current chunk is held
        held = s.num_tokens - bm.base(s.num_tokens - 1)
        assert len(s.table(0)) == (held + 7) // 8
    for s in seqs:
        bm.release(s)
    assert sorted(bm.free) == list(range(200))


def test_page_columns_and_pool_limits():
    assert BlockManager(4, 8, 0, 20).max_blocks(1000) == 3
    assert BlockManager(4, 8, 0, None).max_blocks(1000) == 125
    bm = BlockManager(2, 8, 0, 8)
    s = Sequence(0, 0)
    with pytest.raises(RuntimeError, match="exhausted"):
        bm.extend(s, 0, 24)                                # three chunks in one portion
    slots = StateSlots(1)
    a, b = Sequence(1, 0), Sequence(2, 0)
    slots.allocate(a)
    with pytest.raises(RuntimeError, match="exhausted"):
        slots.allocate(b)
    slots.release(a)
    slots.allocate(b)
    assert a.state_slot == -1 and b.state_slot == 0


def test_engine_stages_every_span_and_the_state_slot(tmp_path):
    small(tmp_path)
    config, source = registry.load_folder(tmp_path, torch.float32)
    config.kv_block_size = 16
    eng = DecodeEngine(config, max_num_seqs=3, max_model_len=200, num_kv_blocks=[9, 12],
                       device="cpu", init_scale=None)
    eng.load_weights(source)
    assert [b.chunk for b in eng.span_blocks] == [24, 40]
    lens = [1, 47, 80]
    eng.add_sequences(lens, [1, 2, 3])
    for step in range(60):
        n = eng.prepare_decode(True)
        h = eng.host_np
        assert n == 3 and sorted(h["state_slots"][:3].tolist()) == [0, 1, 2]
        for i, s in enumerate(eng.seqs):
            pos = lens[i] + step - 1
            assert h["positions"][i] == pos
            for g, chunk in enumerate((24, 40)):
                off = pos % chunk
                assert h["span_lens"][g][i] == off + 1
                assert h["span_slots"][g][i] == s.table(g)[off // 16] * 16 + off % 16
                if eng._bt_dirty:
                    cols = len(s.table(g))
                    assert h["span_tables"][g][i, :cols].tolist() == s.table(g)
                    assert (h["span_tables"][g][i, cols:] == -1).all()
        eng._bt_dirty = False
        for s in eng.seqs:
            s.num_tokens += 1
    first = eng.seqs[0]
    eng.finish(first)
    assert len(eng.state_slots.free) == 1 and first not in eng.seqs
    for s in list(eng.seqs):
        eng.finish(s)
    assert [len(b.free) for b in eng.span_blocks] == [9, 12] and len(eng.state_slots.free) == 3


def test_feeding_a_portion_invalidates_the_staged_tables(tmp_path, monkeypatch):
    """Pages added by a portion must reach the device before the next decode step."""
    small(tmp_path)
    config, source = registry.load_folder(tmp_path, torch.float32)
    config.kv_block_size = 8
    eng = DecodeEngine(config, max_num_seqs=2, max_model_len=200, num_kv_blocks=40, device="cpu",
                       init_scale=None)
    eng.load_weights(source)
    monkeypatch.setattr(type(eng.model), "forward",
                        lambda self, ids, pos: torch.zeros(len(ids), self.stride))
    monkeypatch.setattr(type(eng.model), "project",
                        lambda self, h: torch.zeros(h.shape[0], 51))
    monkeypatch.setattr(eng, "run_step_device", lambda bs: None)
    s = eng.open_sequence()
    for tokens in ([1, 2, 3], [4], [5] * 13, [6], [7] * 9, [8]):
        eng.feed([(s, tokens)])
        if len(tokens) == 1:
            for g in range(2):
                row = eng.graph_vars["span_tables"][g][0].tolist()
                assert row[:len(s.table(g))] == s.table(g)
    with pytest.raises(ValueError, match="at most one entry"):
        eng.feed([(s, [1]), (s, [2])])
    with pytest.raises(ValueError, match="outside"):
        eng.feed([(s, [1] * 400)])


def test_trace_runner_protocol(tmp_path, monkeypatch):
    """Ids become sequences, wanted rows go to files in order, ended requests are given
    back, one 'done' line per step."""
    log = []

    class FakeEngine:
        def open_sequence(self):
            log.append("open")
            return object()

        def feed(self, entries, want):
            return [torch.tensor([[len(t) * 10.0 + p, 1.0] for p in w]).reshape(-1, 2)
                    for (_, t), w in zip(entries, want)]

        def finish(self, seq):
            log.append("finish")

        def device_status(self):
            return 0

    monkeypatch.setattr(trace, "make_engine", lambda *a: FakeEngine())
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]},
                                     {"id": "b", "tokens": [1], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": []}], "end": ["a"]}]
    out = io.StringIO()
    rc = trace.main(["--model", "m", "--out", str(tmp_path), "--max-tokens", "9"],
                    stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"),
                    stdout=out)
    assert rc == 0 and out.getvalue() == "done 0\ndone 1\n"
    data = np.fromfile(tmp_path / "0.f32", "<f4").reshape(-1, 2)
    assert data[:, 0].tolist() == [30.0, 32.0, 10.0]
    assert not (tmp_path / "1.f32").exists()
    assert log == ["open", "open", "finish"]


def test_safetensors_reader_types(tmp_path):
    ints = np.arange(6, dtype="<i4").reshape(2, 3)
    head = json.dumps({"__metadata__": {"a": "b"},
                       "t": {"dtype": "I32", "shape": [2, 3], "data_offsets": [0, 24]},
                       "s": {"dtype": "F32", "shape": [], "data_offsets": [24, 28]}}).encode()
    (tmp_path / "model.safetensors").write_bytes(
        struct.pack("<Q", len(head)) + head + ints.tobytes() + np.float32(2.5).tobytes())
    src = SafetensorsSource(tmp_path)
    assert sorted(src.names()) == ["s", "t"]
    assert src.get("t").tolist() == ints.tolist() and float(src.get("s")) == 2.5


def test_oracle_state_is_carried():
    """The plain recurrence split in two gives what it gives in one piece."""
    rs = np.random.RandomState(0)
    r, k, v = (rs.randn(9, 2, 5) for _ in range(3))
    dec, rate = rs.uniform(0.6, 1, (9, 2, 5)), rs.uniform(0, 1, (9, 2, 5))
    o, s = P.delta_rule(r, k, v, dec, rate)
    o1, s1 = P.delta_rule(r[:4], k[:4], v[:4], dec[:4], rate[:4])
    o2, s2 = P.delta_rule(r[4:], k[4:], v[4:], dec[4:], rate[4:], s1)
    np.testing.assert_allclose(np.concatenate([o1, o2]), o)
    np.testing.assert_allclose(s2, s)


def test_oracle_chunk_edges():
    assert P.visible(23, 0, 24) and not P.visible(24, 23, 24) and P.visible(24, 24, 24)
    assert P.visible(30, 0, None) and not P.visible(3, 4, None)


@pytest.mark.parametrize("name", sorted(P.MODELS))
def test_mistakes_show_in_the_logits(name):
    """The random models of the GPU tests are sharp enough: a chunk one token longer or
    shorter, no token shift, or a state lost on the way moves some position by far more
    than the tolerance there."""
    import copy
    cfg, rank = P.MODELS[name]
    w = P.random_weights(cfg, seed=len(name), rank=rank)
    s = np.random.RandomState(11).randint(0, cfg["vocab"], size=140)
    want = P.logits(cfg, w, s)

    def err(got, ref):
        return (np.sqrt(np.mean((got - ref) ** 2, axis=1)) / np.sqrt(np.mean(want ** 2))).max()
    for d in (1, -1):
        c = copy.deepcopy(cfg)
        c["layers"][0]["mixer"]["left"]["mask"]["size"] += d
        assert err(P.logits(c, w, s), want) > 0.3
    assert err(P.logits(cfg, {**w, "l0.shift": w["l0.shift"] * 0}, s), want) > 0.3
    assert err(P.logits(cfg, w, s[70:])[:20], want[70:90]) > 0.3


def test_a_prefill_that_does_not_fit_gives_everything_back(tmp_path, monkeypatch):
    small(tmp_path)
    config, source = registry.load_folder(tmp_path, torch.float32)
    config.kv_block_size = 8
    eng = DecodeEngine(config, max_num_seqs=2, max_model_len=300, num_kv_blocks=[6, 6],
                       device="cpu", init_scale=None)
    eng.load_weights(source)
    monkeypatch.setattr(type(eng.model), "forward",
                        lambda self, ids, pos: torch.zeros(len(ids), self.stride))
    with pytest.raises(RuntimeError, match="exhausted"):
        eng.prefill([list(range(50)), list(range(40))])
    assert not eng.seqs and len(eng.state_slots.free) == 2
    assert all(len(b.free) == 6 for b in eng.span_blocks)
    # the sizes the engine works out for itself do hold that many tokens
    pages = DecodeEngine.pages_for(config, 90, 2)
    for (chunk, n) in zip((24, 40), pages):
        bm = BlockManager(n, 8, 0, chunk)
        for i, t in enumerate((50, 40)):
            bm.extend(Sequence(i, 0), 0, t)
