"""``python -m openrlhf.cli.trace_run`` -> ``openrlhf_b200.cli.trace_run``."""
import sys

from openrlhf_b200.cli.trace_run import *  # noqa: F401,F403
from openrlhf_b200.cli.trace_run import main

if __name__ == "__main__":
    sys.exit(main())
