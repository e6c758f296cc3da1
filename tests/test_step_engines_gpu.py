"""GPU tests of the 4-bit decoder behind the step interface: the registry builds it and the scheduler serves it."""
import json

import pytest
import torch

from tensorwarp_b200 import checkpoint, registry
from tensorwarp_b200.scheduler import Scheduler
from tensorwarp_b200.state import StateError

pytestmark = pytest.mark.gpu
CONFIG = {"architecture": "TWMarlinQ4", "hidden": 256, "num_heads": 2, "num_kv_heads": 1, "head_dim": 128, "ffn": 512, "vocab": 512,
          "layers": 2, "max_seq": 128, "group_size": 128, "seed": 3}


@pytest.fixture()
def engine(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIG))
    return registry.load(str(tmp_path), max_tokens=96, max_live=4)


def stepwise(engine, prompt, count):
    seq = engine.open()
    token, out = int(engine.step(seq, prompt, [len(prompt) - 1])[0].argmax()), []
    for _ in range(count):
        out.append(token)
        token = int(engine.step(seq, [token], [0])[0].argmax())
    engine.close(seq)
    return out


def test_scheduler_on_the_4_bit_decoder(engine):
    """One sequence at a time; requests that come after another used the cache, prompts in portions, several bursts."""
    assert engine.capacity == 96 and engine.max_live == 1
    prompts = [[5, 9, 200, 31], [7], list(range(40, 75))]
    want = [stepwise(engine, p, 11) for p in prompts]
    sch = Scheduler(engine, portion=8, burst=4)
    requests = [sch.submit(p, 11) for p in prompts]
    assert list(sch.run()) == requests
    assert [r.generated for r in requests] == want


def test_limits(engine):
    seq = engine.open()
    with pytest.raises(StateError):
        engine.open()
    with pytest.raises(StateError):
        engine.step(seq, [1] * 97)
    with pytest.raises(ValueError):
        engine.step(seq, [512])
    with pytest.raises(checkpoint.CheckpointError):
        registry.builder_for(CONFIG)(CONFIG, None, dtype=torch.float32)
