"""Layer-by-layer decoders through the registry, the engine, its cache and its scheduler, against the plain statement of
the whole model in hybrid_oracle.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_oracle as O  # noqa: E402

from nkipy_b200.models import config as C  # noqa: E402
from nkipy_b200.models import registry  # noqa: E402
from nkipy_b200.models.engine import GenerationEngine, Sampling, StepEntry  # noqa: E402
from nkipy_b200.models.hybrid import HybridLM  # noqa: E402
from nkipy_b200.models.kv_cache import OutOfBlocks  # noqa: E402
from nkipy_b200.models.trace import TraceReplay  # noqa: E402
from nkipy_b200.models.weights import hybrid_weight_shapes  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
on_devices = pytest.mark.parametrize("device", DEVICES)
in_dtypes = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
TOL = {torch.float32: 1e-4, torch.bfloat16: 8e-2}


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    """The small tensors of these tests gain nothing from threads and lose a lot when several test processes share cores."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)

# name -> small_config arguments; sizes, orders and branches differ between them
MODELS = {
    "mixed": dict(layers="rara", loop=(1, 3, 3)),
    "loop-first": dict(layers="ar", loop=(0, 1, 2), width=128, groups=1, heads=2, kv_heads=2, dim=32, vdim=64, rdims=32),
    "loop-last": dict(layers="rra", loop=(1, 3, 2), width=72, groups=4, heads=6, kv_heads=1, dim=10, vdim=24, rdims=6,
                      rheads=1, rdim=9, rvdim=70, ff=40, vocab=77),
    "no-loop": dict(layers="aa", width=64, groups=2, heads=3, kv_heads=3, dim=64, vdim=72, rdims=64, scaling=False,
                    softcap=None),
    "one-pass": dict(layers="ra", loop=(0, 2, 1), no_ff=(1,), emb=1.0),
    "no-ff": dict(layers="ra", no_ff=(0, 1), width=40, groups=5, heads=9, kv_heads=1, dim=12, vdim=12, rdims=12,
                  softcap=1.5, vocab=96),
    "recurrent": dict(layers="rr", rheads=2, rdim=132, rvdim=136),
    "odd": dict(layers="ar", width=54, groups=3, heads=2, kv_heads=1, dim=6, vdim=11, rdims=4, rheads=3, rdim=5, rvdim=7,
                ff=33, vocab=61),
}


class Case:
    def __init__(self, name, device, dtype, max_batch=3, blocks=16, seed=1, graph=None):
        self.raw = O.small_config(**MODELS[name])
        self.cfg = registry.architecture_of(self.raw).config(self.raw)
        self.weights = O.small_weights(self.raw, hybrid_weight_shapes(self.cfg), seed)
        self.device, self.dtype = device, dtype
        self.model = HybridLM(self.cfg, self.weights, device=device, dtype=dtype)
        self.engine = GenerationEngine(self.model, max_batch=max_batch, max_seq_len=32 * blocks, num_blocks=blocks,
                                       use_cuda_graph=graph)
        self.scale = None

    def tokens(self, n, seed):
        return torch.randint(0, self.cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def want(self, ids):
        return O.forward(self.raw, self.weights, ids)[0]

    def feed(self, ids, cuts, seq=None):
        """Logits at every position of ids, brought in portions."""
        seq = seq or self.engine.open_request()
        out, lo = [], 0
        for n in cuts:
            out.append(self.engine.run_step([StepEntry(seq, ids[lo:lo + n], range(n))]))
            lo += n
        assert lo == len(ids)
        self.engine.release([seq])
        return torch.cat(out)

    def close(self, got, want, what=""):
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        err = (d.pow(2).mean(-1).sqrt() / want.std()).max().item()
        assert err < TOL[self.dtype], f"{what}: error {err} of the logits' spread"


@on_devices
@in_dtypes
@pytest.mark.parametrize("name", MODELS)
def test_whole_prompts_portions_and_single_tokens(name, device, dtype):
    c = Case(name, device, dtype)
    n = 75
    ids = c.tokens(n, 3)
    want = c.want(ids)
    c.close(c.feed(ids, [n]), want, "whole")
    c.close(c.feed(ids, [2, 2, 31, 1, 1, 28, 10]), want, "portions")
    c.close(c.feed(ids, [40] + [1] * 35), want, "prompt, then single tokens")
    if name in ("mixed", "loop-first"):
        c.close(c.feed(ids, [1] * n), want, "single tokens")
        c.close(c.feed(ids, [2] * 37 + [1]), want, "portions of two")


@on_devices
@pytest.mark.parametrize("name", ["mixed", "loop-last", "one-pass"])
def test_residual_after_every_layer_run(name, device):
    c = Case(name, device, torch.float32)
    ids = c.tokens(21, 5)
    taps = O.forward(c.raw, c.weights, ids)[1]
    s = c.engine.cache.add_sequence(ids)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    _, got = c.model.prefill(t(ids), t(list(range(21))), c.engine.cache.slots_for(s, 0, 21).to(device), c.engine.cache,
                             c.engine.cache.block_table[s.slot:s.slot + 1], t([0]), t([21]), t([21]), 21,
                             return_hidden=True, rows=t([s.slot]))
    assert len(got) == len(taps) == len(c.cfg.layer_runs())
    for i, (a, b) in enumerate(zip(got, taps)):
        assert ((a.double().cpu() - b).abs().max() / b.abs().max()) < 1e-5, f"run {i}"


@on_devices
@in_dtypes
def test_long_prompt_and_long_decoding(device, dtype):
    """Hundreds of tokens: several attention tiles, portions around page and tile borders, far keys."""
    c = Case("mixed", device, dtype)
    n = 420
    ids = c.tokens(n, 8)
    want = c.want(ids)
    c.close(c.feed(ids, [n]), want, "whole")
    c.close(c.feed(ids, [127, 2, 126, 1, 33, 31, 100]), want, "portions")
    c.close(c.feed(ids, [250] + [1] * 170), want, "long decoding")


@on_devices
@in_dtypes
def test_unequal_requests_in_one_batch_match_each_alone(device, dtype):
    c = Case("mixed", device, dtype, max_batch=4, blocks=24)
    lens = [130, 3, 64, 41]
    ids = [c.tokens(n, 20 + i) for i, n in enumerate(lens)]
    want = [c.want(x) for x in ids]
    # portions of some beside single tokens of others; requests pause, end, and their rows and blocks are used again
    plan = [{0: 60, 1: 1}, {0: 1, 1: 1, 2: 33}, {2: 1, 3: 2}, {0: 1, 2: 1, 3: 1}, {1: 1}, {0: 40, 2: 20, 3: 1},
            {0: 1, 3: 1}, {0: 27, 2: 9, 3: 36}]
    at, seqs = {}, {}
    got = {i: [] for i in range(4)}
    for step in plan:
        entries = []
        for i, k in step.items():
            seqs.setdefault(i, None)
            seqs[i] = seqs[i] or c.engine.open_request()
            lo = at.get(i, 0)
            entries.append(StepEntry(seqs[i], ids[i][lo:lo + k], range(k)))
            at[i] = lo + k
        out = c.engine.run_step(entries)
        o = 0
        for i, k in step.items():
            got[i].append(out[o:o + k])
            o += k
    for i, n in enumerate(lens):
        m = sum(len(x) for x in got[i])
        c.close(torch.cat(got[i]), want[i][:m], f"request {i}")
    c.engine.release([s for s in seqs.values()])


@on_devices
@in_dtypes
def test_freed_blocks_and_slots_are_used_again(device, dtype):
    """A pool that holds one and a half requests: every request after the first runs on recycled blocks and slots."""
    c = Case("mixed", device, dtype, max_batch=2, blocks=6)
    for r in range(4):
        a, b = c.tokens(70 + 11 * r, 30 + r), c.tokens(40 + r, 60 + r)
        sa, sb = c.engine.open_request(), c.engine.open_request()
        la = c.engine.run_step([StepEntry(sa, a[:50], range(50)), StepEntry(sb, b[:-5], [0])])
        c.close(la[:50], c.want(a)[:50], f"round {r}")
        outs = []
        for t in range(5):
            lo = len(b) - 5 + t
            outs.append(c.engine.run_step([StepEntry(sb, b[lo:lo + 1], [0]), StepEntry(sa, a[50 + t:51 + t], [])]))
        c.close(torch.cat(outs), c.want(b)[-5:], f"round {r} decoded")
        c.engine.release([sb])
        c.close(c.engine.run_step([StepEntry(sa, a[55:], [len(a) - 56])]), c.want(a)[-1:], f"round {r} rest")
        c.engine.release([sa])
    assert c.engine.cache.allocator.num_free() == 6


@on_devices
def test_step_arguments_are_checked(device):
    c = Case("loop-first", device, torch.float32, max_batch=2, blocks=2)
    s = c.engine.open_request()
    with pytest.raises(ValueError):
        c.engine.run_step([StepEntry(s, [], [])])
    with pytest.raises(ValueError):
        c.engine.run_step([StepEntry(s, [1], []), StepEntry(s, [2], [])])
    with pytest.raises(RuntimeError):
        c.engine.run_step([StepEntry(s, [1] * 65, [])])
    t = c.engine.open_request()
    with pytest.raises(OutOfBlocks):
        c.engine.run_step([StepEntry(s, [1] * 40, []), StepEntry(t, [1], [])])
    assert c.engine.run_step([]) is None


# --------------------------------------------------------------------------- generation, loading, command lines
def greedy_oracle(c, ids, n):
    ids, margins = list(ids), []
    for _ in range(n):
        last = c.want(ids)[-1]
        top = last.topk(2).values
        margins.append(((top[0] - top[1]) / last.std()).item())
        ids.append(int(last.argmax()))
    return ids[-n:], margins


def agrees(got, want, margins, tol):
    for g, w, m in zip(got, want, margins):
        if g != w:
            assert m < tol, f"token {g} instead of {w} at a margin of {m}"
            return                                  # a near tie: the continuations differ from here on


@on_devices
@in_dtypes
@pytest.mark.parametrize("budget", [4096, 16])
def test_greedy_generation_through_the_scheduler(device, dtype, budget):
    c = Case("mixed", device, dtype, max_batch=3, blocks=12)
    c.engine.prefill_chunk_tokens = budget          # 16: every prompt runs in portions
    prompts = [c.tokens(n, 70 + n) for n in (45, 7, 1)]
    for _ in range(2):                              # the second time on recycled rows
        outs = c.engine.generate(prompts, 9)
        for p, o in zip(prompts, outs):
            agrees(o, *greedy_oracle(c, p, 9), TOL[dtype])
    assert not c.engine.active and c.engine.cache.allocator.num_free() == 12


@on_devices
def test_generation_and_steps_share_an_engine(device):
    """A request that is open while others are generated keeps its state and cache."""
    c = Case("mixed", device, torch.float32, max_batch=3, blocks=12)
    ids = c.tokens(60, 90)
    want = c.want(ids)
    s = c.engine.open_request()
    c.engine.run_step([StepEntry(s, ids[:40], [])])
    c.engine.active.pop(s.slot)                     # not a row of the generation below
    c.engine.context_lens[s.slot] = -1
    prompt = c.tokens(20, 91)
    agrees(c.engine.generate([prompt], 6)[0], *greedy_oracle(c, prompt, 6), 1e-4)
    got = [c.engine.run_step([StepEntry(s, [t], [0])]) for t in ids[40:50]]
    c.close(torch.cat(got), want[40:50])
    c.close(c.engine.run_step([StepEntry(s, ids[50:], range(10))]), want[50:])


@on_devices
def test_sampling_follows_the_logits(device):
    c = Case("loop-first", device, torch.float32, max_batch=2, blocks=8)
    prompts = [c.tokens(12, 1), c.tokens(30, 2)]
    greedy = c.engine.generate(prompts, 6)
    assert c.engine.generate(prompts, 6, sampling=Sampling(1.0, top_k=1)) == greedy
    assert c.engine.generate(prompts, 6, sampling=Sampling(0.0)) == greedy
    a = c.engine.generate(prompts, 12, sampling=Sampling(5.0, seed=1))
    b = c.engine.generate(prompts, 12, sampling=Sampling(5.0, seed=2))
    assert a != b and a == c.engine.generate(prompts, 12, sampling=Sampling(5.0, seed=1))


def write_model(folder, name="mixed", seed=4):
    from safetensors.torch import save_file

    raw = O.small_config(**MODELS[name])
    cfg = registry.architecture_of(raw).config(raw)
    w = O.small_weights(raw, hybrid_weight_shapes(cfg), seed)
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(raw))
    save_file(w, str(folder / "model.safetensors"))
    return raw, w


@on_devices
def test_model_folder_loads_by_its_architecture(device, tmp_path):
    raw, w = write_model(tmp_path / "m")
    model = registry.load_model(str(tmp_path / "m"), device=device, dtype=torch.float32)
    assert isinstance(model, HybridLM) and model.cfg.loop == C.LoopSpec(1, 3, 3)
    assert model.cfg.param_count() == sum(t.numel() for t in w.values())
    eng = GenerationEngine(model, max_batch=1, max_seq_len=64)
    ids = list(range(40))
    s = eng.open_request()
    got = eng.run_step([StepEntry(s, ids, range(40))])
    want = O.forward(raw, w, ids)[0]
    assert ((got.double().cpu() - want).abs().max() / want.std()) < 1e-3


def test_config_reader_rejects_what_it_does_not_know():
    raw = O.small_config(**MODELS["mixed"])
    for change in (lambda r: r.update(architecture="Other"), lambda r: r["layers"][0].update(type="other"),
                   lambda r: r["layers"][0].update(mlp={"kind": "other", "ff": 8})):
        bad = json.loads(json.dumps(raw))
        change(bad)
        with pytest.raises(ValueError):
            registry.architecture_of(bad).config(bad)


def test_registry_reads_other_families():
    hf = {"architectures": ["Qwen3MoeForCausalLM"], "hidden_size": 64, "num_hidden_layers": 2, "num_attention_heads": 4,
          "num_key_value_heads": 2, "head_dim": 32, "vocab_size": 99, "num_experts": 4, "num_experts_per_tok": 2,
          "moe_intermediate_size": 48, "intermediate_size": 7, "rms_norm_eps": 1e-4}
    cfg = registry.architecture_of(hf).config(hf)
    assert (cfg.num_experts, cfg.top_k, cfg.moe_intermediate_size, cfg.intermediate_size) == (4, 2, 48, 0)
    assert cfg.qk_norm and cfg.rms_eps == 1e-4 and cfg.num_layers == 2
    hf = {"architectures": ["GptOssForCausalLM"], "num_hidden_layers": 4, "num_local_experts": 8, "intermediate_size": 96,
          "sliding_window": 16}
    cfg = registry.architecture_of(hf).config(hf)
    assert (cfg.num_experts, cfg.moe_intermediate_size, cfg.sliding_window, len(cfg.layer_types)) == (8, 96, 16, 4)


@on_devices
def test_trace_command_replays_steps(device, tmp_path):
    raw, w = write_model(tmp_path / "m", "loop-last")
    out = tmp_path / "out"
    out.mkdir()
    g = torch.Generator().manual_seed(5)
    a, b = (torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for n in (50, 9))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:45], "want": [3, 44]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:4], "want": []}, {"id": "a", "tokens": a[45:46], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[4:5], "want": [0]}, {"id": "a", "tokens": a[46:47], "want": [0]}],
              "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[5:], "want": [3]}, {"id": "a", "tokens": a[:20], "want": [19]}],
              "end": ["a", "b"]}]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                          "--out", str(out), "--max-tokens", "128", "--device", device],
                         input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=900)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
    wa, wb = O.forward(raw, w, a)[0], O.forward(raw, w, b)[0]
    for n, want in ((0, wa[[3, 44]]), (2, torch.stack([wb[4], wa[46]])), (3, torch.stack([wb[8], wa[19]]))):
        got = torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, raw["vocab"])
        assert ((got.double() - want).abs().max() / want.std()) < 1e-3


@on_devices
def test_generation_command_line(device, tmp_path):
    write_model(tmp_path / "m")
    env = dict(os.environ, PYTHONPATH=ROOT)
    if device == "cpu":
        env["CUDA_VISIBLE_DEVICES"] = ""
    cmd = [sys.executable, "-m", "nkipy_b200.models.runner", "--model", str(tmp_path / "m"), "--batch", "2",
           "--prompt-len", "12", "-n", "4", "--max-seq-len", "96"]
    for extra in ([], ["--dtype", "float32", "--temperature", "0.8", "--top-k", "5"]):
        res = subprocess.run(cmd + extra, capture_output=True, text=True, timeout=600, env=env, cwd=ROOT)
        assert res.returncode == 0 and "Decode tokens/sec" in res.stdout, res.stderr[-2000:]


def test_replay_returns_what_requests_hold():
    c = Case("loop-first", "cpu", torch.float32, max_batch=4, blocks=4)
    r = TraceReplay(c.engine)
    for n in range(6):
        out = r.step({"step": n, "entries": [{"id": f"r{n}", "tokens": c.tokens(100, n), "want": [99]}], "end": [f"r{n}"]})
        assert out.shape == (1, c.cfg.vocab_size) and out.dtype == torch.float32
    assert not r.live and c.engine.cache.allocator.num_free() == 4
