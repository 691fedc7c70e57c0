"""Mumilorn generation: pre-norm layers of gated linear attention, and of windowed attention beside RWKV-style time mixing,
with dense or routed feed-forwards.

    python examples/models/mumilorn/mumilorn.py -n 64 --batch 8                      # random weights
    python examples/models/mumilorn/mumilorn.py --model /path/to/model -n 64         # config.json + model.safetensors
    python examples/models/mumilorn/mumilorn.py --tiny --dtype float32 -n 8          # quick functional run
"""
import argparse
import os
import sys

sys.path.insert(0, os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "..", ".."))

from nkipy_b200.models import runner  # noqa: E402
from nkipy_b200.models.config import mumilorn_shape  # noqa: E402


def main():
    if "--model" in sys.argv:
        return runner.main()
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    runner.add_common_args(ap)
    cfg = mumilorn_shape(2048, layers=12, heads=16, kv_heads=4, ff=5632, experts=16, top=4, expert_ff=704, groups=4, keep=2)
    return runner.run_generation(cfg, ap.parse_args())


if __name__ == "__main__":
    sys.exit(main())
