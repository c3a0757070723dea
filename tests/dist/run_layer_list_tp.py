"""Two tensor-parallel gloo ranks serve a checkpoint in portions; every rank compares with the expected logits."""
import os
import sys

import torch
import torch.distributed as dist

HERE = os.path.dirname(os.path.abspath(__file__))
sys.path[:0] = [os.path.dirname(os.path.dirname(HERE)), os.path.dirname(HERE)]

from mindformers_b200.models import AutoModel  # noqa: E402
from mindformers_b200.parallel import parallel_state as ps  # noqa: E402
from mindformers_b200.serving.trace import build_engine  # noqa: E402
from oracles import cases  # noqa: E402

dist.init_process_group("gloo")
ps.initialize_model_parallel(tensor_model_parallel_size=dist.get_world_size())
model = AutoModel.from_pretrained(sys.argv[1], dtype="float32", device="cpu", strict=True,
                                  tensor_model_parallel_size=dist.get_world_size()).eval()
want = torch.load(sys.argv[2])
toks = cases.tokens(want.shape[0], want.shape[1], seed=1)
got = cases.run_schedule(build_engine(model, 64), {"a": toks}, [{"a": 23}, {"a": 2}, {"a": 1}, {"a": want.shape[0] - 26}])["a"]
err = cases.worst(got, want)
dist.destroy_process_group()
assert err < 2e-5, err
