"""Host-side logic of the matrix-memory / grouped-attention decoder: configuration, registry, parameter
layouts, sequence state, split rules, argument validation of its kernels."""
import ctypes
import json

import pytest
import torch

import mutolix_plain as P
import tulezen_plain as T
from energonai_b200 import _lib, registry
from energonai_b200.attention import pick_group_nsplit
from energonai_b200.gemm import xielu_params
from energonai_b200.model import GenerationModel, LayeredDecoder, RecurrentState, RingCache, SandwichDecoder, SandwichDecoderConfig, SequenceState
from energonai_b200.model.grouped_attention import padded_head
from energonai_b200.utils import processing_Mutolix


def config():
    return P.make_config([P.memory_layer(3, 20, 28, 7.0), P.attention_layer(6, 2, 12, 20, 0.3, 0.2, 5, ff=44), P.memory_layer(1, 8, 12, 3.0, ff=20),
                          P.attention_layer(4, 4, 36, 8, 0.2, 0.5, 7, v_mix=False), P.attention_layer(2, 2, 9, 20, 0.4, 0.1, 1)], width=52, vocab=83)


def test_configuration_reads_every_size_and_rejects_what_it_does_not_know():
    c = SandwichDecoderConfig.from_dict(config())
    assert (c.vocab, c.width, c.eps, c.embed_scale, len(c.layers)) == (83, 52, 2e-5, 1.7, 5)
    m = c.layers[0].mixer
    assert (m.heads, m.dim, m.vdim, m.gate_cap) == (3, 20, 28, 7.0) and c.layers[0].mlp is None and c.layers[2].mlp.ff == 20
    a = c.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.temp_coef, a.temp_every, a.v_mix) == (6, 2, 12, 20, 0.3, 0.2, 5, True)
    assert [c.layers[i].mixer.v_from for i in (1, 3, 4)] == [None, None, 1]
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][1]["mlp"].update(kind="moe"),
                   lambda d: d["layers"][1]["mixer"].update(kv_heads=4), lambda d: d["layers"][4]["mixer"].update(vdim=12),
                   lambda d: d["layers"][0]["mixer"].update(gate_cap=0), lambda d: d["layers"][1]["mixer"]["q_temp"].update(every=0),
                   lambda d: d["layers"][1]["mixer"].update(mask={"size": 8}), lambda d: d["layers"][0]["mixer"].update(conv=4)):
        d = json.loads(json.dumps(config()))
        change(d)
        with pytest.raises(ValueError):
            SandwichDecoderConfig.from_dict(d)
    d = config()
    d["layers"][1]["mixer"].update(mask=None)               # says that there is none
    del d["layers"][1]["mixer"]["q_temp"]
    assert SandwichDecoderConfig.from_dict(d).layers[1].mixer.temp_every == 0
    del d["layers"][1]["mixer"]["scale"]
    with pytest.raises(KeyError):
        SandwichDecoderConfig.from_dict(d)


def test_registry_knows_the_design():
    assert "Mutolix" in registry.architectures()
    model = registry.build_model("Mutolix", config_dict=config(), dtype=torch.float32)
    assert isinstance(model, SandwichDecoder) and isinstance(model, LayeredDecoder) and isinstance(model, GenerationModel)


def test_head_padding_is_common_to_layers_that_share_values():
    assert padded_head([40, 64], torch.bfloat16) == 64 and padded_head([65], torch.float16) == 128
    assert padded_head([129], torch.bfloat16) is None and padded_head([8], torch.float32) is None
    cfg = P.make_config([P.attention_layer(2, 1, 16, 24, 0.3, 0.1, 4), P.attention_layer(2, 1, 100, 24, 0.3, 0.1, 4),
                         P.attention_layer(2, 1, 16, 24, 0.3, 0.1, 4, v_mix=False)], width=16, vocab=16)
    m = registry.build_model("Mutolix", config_dict=cfg, dtype=torch.bfloat16)
    assert [b.mixer.dv for b in m.layers] == [128, 128, 64]
    m = registry.build_model("Mutolix", config_dict=cfg, dtype=torch.float32)
    assert [(b.mixer.dk, b.mixer.dv) for b in m.layers] == [(16, 24), (104, 24), (16, 24)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_parameters_in_kernel_layout_hold_the_checkpoint(tmp_path, dtype):
    cfg = config()
    t = P.make_tensors(cfg, 3)
    T.save_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    model = registry.load_model(str(tmp_path), dtype=dtype, device="cpu")
    f = lambda name: t[name].float()
    g = torch.Generator().manual_seed(1)
    W, w = model.hidden_size, cfg["width"]
    h = torch.zeros(4, W)
    h[:, :w] = torch.randn(4, w, generator=g)
    hs = h[:, :w]

    def heads(y, n, padded, dim):
        y = y.view(4, n, padded)
        assert float(y[..., dim:].abs().sum()) == 0
        return y[..., :dim].reshape(4, -1)
    close = lambda a, b: torch.allclose(a, b, atol=2e-5)
    for i, ly in enumerate(cfg["layers"]):
        blk, m, p = model.layers[i], ly["mixer"], f"l{i}."
        at = blk.mixer
        y = h @ at.in_proj.float().T + at.bias.float()
        if ly["type"] == "mlstm":
            q, k, v, o, rg = y[:, :at.tail].split(at.splits, 1)
            gates = y[:, at.tail:]
            for got, name, pad, dim in ((q, "q", at.dk, m["dim"]), (k, "k", at.dk, m["dim"]), (v, "v", at.dv, m["vdim"]), (o, "g", at.dv, m["vdim"])):
                assert close(heads(got, m["heads"], pad, dim), hs @ f(p + "mix." + name).T)
            H = m["heads"]
            assert close(gates[:, :H], hs @ f(p + "mix.i").T) and close(gates[:, H:2 * H], hs @ f(p + "mix.f").T)
            assert torch.equal(at.gate_bias, torch.stack([f(p + "mix.i.b"), f(p + "mix.f.b")])) and at.gate_bias.dtype == torch.float32
        else:
            q, k, v, rg = y.split(at.splits, 1)
            for got, name, n, pad, dim in ((q, "q", m["heads"], at.dk, m["dim"]), (k, "k", m["kv_heads"], at.dk, m["dim"]),
                                           (v, "v", m["kv_heads"], at.dv, m["vdim"])):
                assert close(heads(got, n, pad, dim), hs @ f(p + "mix." + name).T + f(p + f"mix.{name}.b"))
            assert torch.equal(at.r1, f(p + "mix.r1")) and torch.equal(at.r2, f(p + "mix.r2")) and at.r1.dtype == torch.float32
            assert at.v_from is None or float(at.vmix) == float(t[p + "mix.vmix"])
        for s in ("1", "2") if ly["mlp"] else ("1",):
            out = getattr(blk, "out" + s)
            assert out.dtype == torch.float32 and torch.equal(out[:w], f(p + f"norm{s}b") * f(p + "ls" + s)) and float(out[w:].abs().sum()) == 0
        assert close(rg[:, :w], hs @ f(p + "rg1").T + f(p + "rg1.b")) and float(rg[:, w:].abs().sum()) == 0
        z = torch.zeros(4, m["heads"], at.dv)
        z[..., :m["vdim"]] = torch.randn(4, m["heads"], m["vdim"], generator=g)
        assert close((z.view(4, -1) @ at.out_proj.float().T)[:, :w], z[..., :m["vdim"]].reshape(4, -1) @ f(p + "mix.o").T)
        if ly["mlp"]:
            u = h @ blk.mlp.up.float().T + blk.mlp.bias.float()
            ff = ly["mlp"]["ff"]
            assert close(u[:, :ff], hs @ f(p + "mlp.up").T) and close(u[:, blk.mlp.ff_padded:][:, :w], hs @ f(p + "rg2").T + f(p + "rg2.b"))
            want = torch.nn.functional.softplus(f(p + "mlp.act"))
            assert torch.allclose(blk.mlp.act, want + torch.tensor([0.0, 0.5]))
        else:
            assert blk.mlp is None


def test_checkpoint_conversion_complains_about_missing_surplus_and_misshapen_tensors():
    cfg = config()
    t = P.make_tensors(cfg, 3)
    model = registry.build_model("Mutolix", config_dict=cfg, dtype=torch.float32)
    processing_Mutolix(t, model)
    processing_Mutolix({k: v for k, v in t.items() if k != "l1.mix.vmix"}, model)       # the first layer's is not used
    for name in ("l0.mix.f", "l4.mix.vmix", "l1.ls2", "l2.rg2.b"):
        with pytest.raises(KeyError, match="lacks"):
            processing_Mutolix({k: v for k, v in t.items() if k != name}, model)
    with pytest.raises(KeyError, match="l0.norm2"):
        processing_Mutolix(dict(t, **{"l0.norm2": t["l0.norm1"]}), model)
    with pytest.raises(ValueError, match="l1.mix.q"):
        processing_Mutolix(dict(t, **{"l1.mix.q": t["l1.mix.q"][:-1]}), model)


def test_xielu_numbers():
    a = xielu_params(0.0, 1.0)
    assert torch.allclose(a, torch.tensor([0.6931472, 1.8132617])) and a.dtype == torch.float32


def test_state_of_both_kinds_is_prepared_used_again_kept_and_forked():
    s = SequenceState({0: RecurrentState([(2, 4, 8), (2, 4), (2,)]), 1: RingCache(16)})
    dev = torch.device("cpu")
    s.begin([2, 0, 1], 6, 3, torch.float32, dev)
    S, n, m = s.caches[0].tensors
    assert S.shape == (3, 2, 4, 8) and n.shape == (3, 2, 4) and m.shape == (3, 2) and S.dtype == torch.float32
    assert s.capacity() == 9
    for t in (S, n, m, s.caches[1].buf):
        t.copy_(torch.arange(3.).view(3, *[1] * (t.dim() - 1)).expand_as(t))
    two = s.fork([1])
    s.keep([0, 2])
    assert [float(t.mean()) for t in two.caches[0].tensors] == [1.0, 1.0, 1.0] and float(two.caches[1].buf.mean()) == 1.0
    assert s.caches[0].tensors[2][:, 0].tolist() == [0.0, 2.0] and s.caches[1].buf[:, 0, 0].tolist() == [0.0, 2.0]
    two.caches[0].tensors[0].fill_(9.0)
    assert float(s.caches[0].tensors[0].max()) == 2.0                       # memory of its own
    before = s.caches[0].pointers()
    s.begin([0, 0], 4, 1, torch.float32, dev)
    assert s.caches[0].pointers() == before and all(float(t.abs().sum()) == 0 for t in s.caches[0].tensors)      # used again, from zero
    s.ensure(40)
    assert s.capacity() >= 40 and s.caches[0].room() is None
    s.begin([0], 4, 1, torch.float32, dev)
    assert s.caches[0].tensors[0].shape[0] == 1


def test_caches_of_the_model():
    m = registry.build_model("Mutolix", config_dict=config(), dtype=torch.bfloat16)
    kinds = [type(m.state.caches[i]) for i in range(5)]
    assert kinds == [RecurrentState, RingCache, RecurrentState, RingCache, RingCache]
    assert m.state.caches[0].shapes == [(3, 64, 32), (3, 64), (3,)] and m.state.caches[1].width == 2 * 2 * 64


def test_split_rule_of_head_groups():
    assert pick_group_nsplit(1, 1, 100) == 1 and pick_group_nsplit(1, 1, 1 << 20) == 64
    assert pick_group_nsplit(1, 8, 1024) == 4                    # never under 256 keys each
    assert pick_group_nsplit(64, 16, 4096) <= 2                  # a full machine is hardly split
    for b, u, k in ((64, 4, 2048), (16, 8, 4096)):
        assert b * u * pick_group_nsplit(b, u, k) >= 2 * 148


def test_kernels_validate_before_any_cuda_call():
    L = _lib.lib()
    buf = ctypes.create_string_buffer(64)
    a = (ctypes.addressof(buf) + 15) & ~15
    B16, F16, F32 = _lib.BF16, _lib.F16, _lib.F32
    err = _lib.last_error
    stream = lambda **k: L.eb_stream_update(k.get("src"), 8, 1.0, k.get("y"), 8, k.get("gate"), 8, k.get("wo"), a, 8, k.get("wn"), k.get("h"), 8, 1e-5,
                                            1, k.get("n2", 8), 8, B16, None)
    assert stream(y=a) == -1 and "weight" in err()
    assert stream(wn=a) == -1 and stream(src=a, gate=a) == -1 and stream() == -1
    assert stream(src=a, n2=12) == -1 and "multiple of 8" in err()
    parts = lambda cols=0, act=None, tail_col=8, tail=a, ldt=8: L.eb_gemm_parts(a, 8, a, 8, a, 8, None, 4, 16, 8, cols, act, tail_col, tail, ldt, B16, 0, None, 0, None)
    assert parts(cols=4, act=a) == -1 and "multiple of 8" in err()
    assert parts(tail_col=12) == -1 and "tail" in err() and parts(ldt=4) == -1
    inputs = lambda dk=8, qc=8, every=0, vmix=None: L.eb_attention_inputs(a, 64, 1, 1, dk, 8, a, qc, a, 8, 1e-5, 0.0, every, vmix, None, 0, 0, a, 8, a, 8, 8, a, 8, 8,
                                                                          4, 1, 1, None, None, B16, None)
    assert inputs(dk=12) == -1 and inputs(qc=9) == -1 and inputs(every=-1) == -1 and inputs(vmix=a) == -1
    scan = lambda fn, dk=64, dv=8, cap=1.0, dtype=B16: fn(a, a, a, 64, a, 2, a, a, cap, 1.0, None, a, 8, a, a, a, 1, 1, 1, dk, dv, dtype, None)
    assert scan(L.eb_memory_scan, dk=12) == -1 and scan(L.eb_memory_scan, cap=0.0) == -1 and "cap" in err()
    assert scan(L.eb_memory_chunks, dk=96) == -1 and "64 or 128" in err()
    assert scan(L.eb_memory_chunks, dtype=F16) == -1 and "bf16" in err() and scan(L.eb_memory_chunks, dv=12) == -1
    step = lambda count=8: L.eb_memory_step(a, a, a, a, 64, a, 2, a, a, 1.0, 1.0, a, count, 1e-5, a, 8, a, a, a, 1, 1, 8, 8, B16, None)
    assert step(count=9) == -1
    assert L.eb_head_norm_gate(a, 8, a, 8, a, 1e-5, a, 8, 1, 1, 12, 8, B16, None) == -1
    group = lambda heads=4, kv=2, d=64, dtype=B16, nsplit=1: L.eb_attention_group_decode(a, a, a, a, 256, 640, 128, 640, 128, 256, 1, heads, kv, d, 5, a, None, None,
                                                                                         None, 1, 1.0, dtype, nsplit, None, 0, None)
    assert group(heads=3) == -1 and "share" in err()
    assert group(d=96) == -1 and group(dtype=F32) == -1 and group(nsplit=2) == -1 and "scratch" in err()
    assert L.eb_attention_group_decode_scratch_bytes(2, 40, 2, 64, 3) == 65536 + 2 * 2 * 2 * 3 * 16 * 66 * 4
    assert L.eb_attention_group_decode_scratch_bytes(2, 40, 2, 64, 1) == 0
    biased = lambda group=1, n=264: L.eb_attention_prefill_biased_tc(a, a, a, a, None, *[64] * 8, 0, 1, 2, group, 8, 8, 64, 0, a, n, 1, 0.1, B16, None)
    assert biased(group=3) == -1 and biased(n=100) == -1 and "bias table" in err()
    assert L.eb_attention_plain(a, a, a, a, *[8] * 12, 1, 3, 2, 1, 8, 8, 0, 4, None, None, None, None, 0, 1.0, F32, None) == -1
    assert L.eb_attention_plain(a, a, a, a, *[8] * 12, 1, 2, 2, 1, 8, 8, 0, 4, None, None, a, None, 0, 1.0, F32, None) == -1 and "bias" in err()
    assert L.eb_distance_bias(None, a, 1, 4, a, None) == -1
    assert L.eb_gemm_f32(a, 8, 0, a, 8, 0, a, 8, 0, 1, 8, 8, 2, None, None, a, 0, None, None) == -1
